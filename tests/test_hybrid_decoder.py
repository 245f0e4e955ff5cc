"""Duvivik on the hybrid decoder: kernels and mixers against the plain statement in ``duvivik_oracle.py``, then whole models
through the generator's step function, the paged state cache, the batching engine and the command line."""
import copy
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import duvivik_oracle as O

from pmetal_b200.models.architectures import build_model, family_of
from pmetal_b200.models.generation import GraphedDecoder
from pmetal_b200.models.hybrid_decoder import PRESETS, HybridArgs, HybridDecoderLM
from pmetal_b200.models.kv_cache import BLOCK
from pmetal_b200.models.loader import load_pretrained, save_pretrained
from pmetal_b200.models.state_cache import CacheSpec, StateCache, split_groups

gpu = pytest.mark.gpu
FP32 = 3e-5          # worst row of fp32 models, see ``err``


# ------------------------------------------------------------------------------------------- models of the tests
def attn(heads, dim, rot, vdim, rank, base=10000.0, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot) ** -0.5,
         "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def ssm(heads, vdim, state, groups, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def config(layers, width=48, vocab=101, alpha=2.0, scale=0.7, eps=1e-5):
    """layers: (mixer dict, ff or None, limit)."""
    return {"architecture": "Duvivik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "postln_alpha": alpha,
            "norm": {"eps": eps},
            "layers": [{"type": "mamba2" if "state" in m else "latent_attention", "mixer": m,
                        "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": lim}} for m, ff, lim in layers]}


MODELS = {
    # own latents at two places, two readers of different sizes, a state-space layer with and without feed-forward
    "mixed": config([(attn(3, 16, 8, 24, 40), 72, 1.2), (ssm(6, 20, 16, 3, 4, 2), None, 0), (attn(5, 24, 8, 16, 40, kv_from=0), None, 0),
                     (attn(2, 32, 16, 32, 64, base=500.0), 40, 0.8), (ssm(4, 32, 48, 1, 3, 4), 56, 2.0),
                     (attn(4, 8, 16, 40, 64, base=500.0, kv_from=3), 24, 1.0)]),
    # sizes that are not multiples of what the fast kernels copy at a time
    "odd": config([(ssm(3, 7, 10, 3, 5, 3), 30, 1.5), (attn(3, 5, 6, 9, 21), 33, 1.1), (ssm(2, 9, 5, 1, 2, 1), None, 0),
                   (attn(1, 11, 6, 3, 21, kv_from=1), None, 0)], width=42, vocab=77, alpha=1.3, scale=1.9, eps=1e-3),
    # everything that may be one
    "ones": config([(ssm(1, 16, 16, 1, 1, 1), None, 0), (attn(1, 16, 16, 16, 16), 16, 3.0), (ssm(2, 8, 1, 1, 4, 1), 16, 0.5)],
                   width=32, vocab=40, alpha=1.0, scale=1.0),
    # many heads (two row tiles), heads wider than the expanded kernels take, a state that needs the scan everywhere
    "wide": config([(attn(20, 16, 16, 16, 128), 64, 1.0), (attn(2, 120, 32, 136, 72), None, 0), (ssm(2, 64, 144, 2, 4, 2), None, 0),
                    (ssm(2, 72, 128, 2, 4, 1), None, 0)], width=64, vocab=90),
}


def random_weights(cfg, seed=0):
    """bf16-representable weights; queries and keys are large enough for peaked attention, step sizes small enough for
    states that live long."""
    g = torch.Generator().manual_seed(seed)
    m = HybridDecoderLM(HybridArgs.from_dict(cfg), device="meta")
    sd = {}
    for name, shape, _, _ in m.named_weights():
        leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
        n = lambda s=1.0: torch.randn(shape, generator=g) * s      # noqa: E731
        u = lambda a, b: torch.rand(shape, generator=g) * (b - a) + a      # noqa: E731
        if leaf == "mix.A_log":
            t = u(-2.0, 1.5)
        elif leaf == "mix.dt_bias":
            t = u(-4.0, 0.0)
        elif leaf.endswith("norm") or leaf in ("norm1", "norm2", "mix.D"):
            t = u(0.5, 1.5)
        elif leaf.endswith(".b"):
            t = n(0.2)
        elif leaf == "mix.conv":
            t = n(0.7)
        elif leaf in ("mix.q", "mix.uk"):
            t = n(1.8 * shape[1] ** -0.5)
        elif leaf == "embed":
            t = n()
        else:
            t = n(shape[1] ** -0.5)
        sd[name] = t.to(torch.bfloat16)
    return sd


_BUILT = {}


def built(name, dtype=torch.float32, device="cuda"):
    """(config, oracle weights, model) of one of MODELS, cached."""
    key = (name, dtype, device)
    if key not in _BUILT:
        cfg = MODELS[name]
        sd = random_weights(cfg)
        m = build_model(cfg, dtype, device)
        assert m.load_hf_state_dict(sd) == []
        _BUILT[key] = (cfg, {k: v.double() for k, v in sd.items()}, m.eval())
    return _BUILT[key]


_ORACLE = {}


def oracle(name, tokens):
    key = (name, tuple(tokens))
    if key not in _ORACLE:
        cfg = MODELS[name]
        sd = {k: v.double() for k, v in random_weights(cfg).items()}
        _ORACLE[key] = O.forward(list(tokens), sd, cfg)[0]
    return _ORACLE[key]


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def err(got, want):
    """Per-row root mean square of the difference (mean taken off) over that of the expected logits; worst row."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()).max())


def bf16_bound(run, want):
    """Tolerance of a bf16 comparison: twice what rounding the oracle's own projections and activations to bf16 does to it
    in the worst row (``run`` recomputes it), plus a little for rows that rounding happens to leave alone."""
    with O.rounding():
        return 2 * err(run(), want) + 5e-3


_BOUND = {}


def bound(name, toks, dtype):
    if dtype == torch.float32:
        return FP32
    key = (name, tuple(toks))
    if key not in _BOUND:
        cfg = MODELS[name]
        sd = {k: v.double() for k, v in random_weights(cfg).items()}
        _BOUND[key] = bf16_bound(lambda: O.forward(list(toks), sd, cfg)[0], oracle(name, toks))
    return _BOUND[key]


def generator(model, blocks=64, max_seqs=4, **kw):
    from pmetal_b200.models.generation import Generator
    return Generator(model, cache=model.new_cache(blocks, max_seqs=max_seqs), **kw)


def feed(gen, seq, toks, sizes):
    """Logits of all positions of ``toks`` fed in portions of the given sizes (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        out.append(gen.step([seq], [toks[at:at + n]], [list(range(n))]).float().cpu())
        at, k = at + n, k + 1
    return torch.cat(out)


# ------------------------------------------------------------------------------------------- host side (no GPU)
def test_registry_and_configuration():
    cfg = MODELS["mixed"]
    assert family_of(cfg) == "hybrid" and family_of({"model_type": "duvivik"}) == "hybrid"
    assert family_of({"model_type": "qwen3"}) == "fast" and family_of({"model_type": "nemotron_h"}) == "nemotron_h"
    a = HybridArgs.from_dict(cfg)
    assert (a.vocab_size, a.hidden_size, a.num_hidden_layers, a.residual_alpha, a.embed_scale) == (101, 48, 6, 2.0, 0.7)
    assert a.to_hf_dict() == cfg and a.to_hf_dict() is not cfg
    m = build_model(cfg, torch.float32, "cpu")
    assert isinstance(m, HybridDecoderLM)
    assert [l.mixer.cache_spec().page_width for l in m.layers] == [56, 0, 0, 88, 0, 0]
    with pytest.raises(RuntimeError, match="CUDA"):
        m(torch.tensor([1, 2]))


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=48), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "norm parts"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4), "rot"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0].update(type="window"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_bad_configurations_are_refused(change, what):
    c = copy.deepcopy(MODELS["mixed"])
    change(c)
    with pytest.raises(ValueError, match=what):
        HybridArgs.from_dict(c)


def test_checkpoint_round_trip(tmp_path):
    cfg = MODELS["odd"]
    sd = random_weights(cfg, 3)
    m = build_model(cfg, torch.bfloat16, "cpu")
    m.load_hf_state_dict(sd)
    save_pretrained(m, str(tmp_path))
    for dtype in (torch.bfloat16, torch.float32):
        back, args, mdir = load_pretrained(str(tmp_path), dtype)
        assert mdir == str(tmp_path) and args.to_hf_dict() == cfg
        got = back.hf_state_dict()
        assert set(got) == set(sd) and all(torch.equal(got[k], sd[k]) for k in sd)
    missing = {k: v for k, v in sd.items() if k != "l1.mix.dkv.norm"}
    with pytest.raises(KeyError, match="dkv.norm"):
        m.load_hf_state_dict(missing)
    with pytest.raises(ValueError, match="shape"):
        m.load_hf_state_dict(dict(sd, **{"l0.mix.D": torch.zeros(4)}))


def test_state_cache_bookkeeping():
    specs = [CacheSpec(page_width=16), CacheSpec(slots={"conv": ((2, 3), None), "state": ((4,), torch.float32)}), CacheSpec()]
    c = StateCache(specs, 4, 2, torch.bfloat16, "cpu")
    assert list(c.pages) == [0] and c.pages[0].shape == (5, BLOCK, 16) and c.slots[1]["state"].dtype == torch.float32
    assert c.slots[1]["conv"].shape == (3, 2, 3) and (c.scratch_block, c.scratch_slot) == (4, 2)
    c.add_sequence(7)
    m = c.prepare([7], [70])
    assert m.state_slots.tolist() == [c.slot_of[7]] and m.seq_of.tolist() == [0] * 70 and c.num_free() == 2
    c.slots[1]["state"][c.slot_of[7]] = 3.0
    c.pages[0][c.seqs[7].blocks[1]] = 5.0
    c.fork(7, 8)
    assert not c.can_admit() and c.slots[1]["state"][c.slot_of[8]].tolist() == [3.0] * 4
    with pytest.raises(MemoryError, match="slots"):
        c.add_sequence(9)
    with pytest.raises(MemoryError, match="slots"):
        c.fork(7, 9)
    c.prepare([8], [1])                                    # the shared tail block is copied before it is written
    assert c.seqs[8].blocks[0] == c.seqs[7].blocks[0] and c.seqs[8].blocks[1] != c.seqs[7].blocks[1]
    assert float(c.pages[0][c.seqs[8].blocks[1]].float().min()) == 5.0
    with pytest.raises(ValueError, match="absorbed"):
        c.truncate(8, 64)
    m = c.prepare([8, 7], [2, 40])
    assert m.seq_of.tolist() == [0, 0] + [1] * 40 and m.positions.tolist() == [71, 72] + list(range(70, 110))
    c.free_sequence(7)
    c.free_sequence(8)
    assert c.num_free() == 4 and sorted(c.free_slots) == [0, 1]
    c = StateCache(specs[:1], 4, 2, torch.bfloat16, "cpu")             # nothing per sequence: any number of them
    for i in range(5):
        c.add_sequence(i)
    assert c.can_truncate and c.can_admit() and c.bytes_per_token() == 32 and set(c.slot_of.values()) == {0}


def test_split_groups():
    c = StateCache([CacheSpec(page_width=16)], 16, 4, torch.float32, "cpu")
    for i in range(4):
        c.add_sequence(i)
    c.prepare([2], [100])
    meta = c.prepare([0, 1, 2, 3], [1, 40, 2, 17])
    s, l = split_groups(meta, 16)
    assert (s.n, s.n_tok, s.max_q, s.max_kv) == (2, 3, 2, 102) and s.q_start.tolist() == [0, 41] and s.c_start.tolist() == [0, 1]
    assert s.tok_rows.tolist() == [0, 41, 42]
    assert s.seq_lens.tolist() == [1, 102] and s.state_slots.tolist() == [c.slot_of[0], c.slot_of[2]]
    assert (l.n, l.max_q) == (2, 40) and l.host == [(1, 1, 40, 40), (3, 43, 17, 17)]
    a, b = split_groups(meta, 64)
    assert b is None and a.n == 4 and a.block_table is meta.block_table
    a, b = split_groups(meta, 0)
    assert a is None and b.n == 4


def test_captured_step_tables_follow_recycled_blocks():
    """A sequence whose table has the same ends and length as the row's previous owner still gets its own table."""
    g = object.__new__(GraphedDecoder)
    g.cache = StateCache([CacheSpec(page_width=16)], 8, 2, torch.float32, "cpu")
    g.state_slots, g.pad_block = g.cache.slot_of, 8
    st = {"h64": torch.zeros(4, dtype=torch.int64), "h32": torch.zeros(4 + 16 + 2, dtype=torch.int32)}
    g._fill(st, 2, 8, [0], [200], [201], [[1, 2, 3, 4]], [5], [1])
    g._fill(st, 2, 8, [0], [200], [201], [[1, 3, 2, 4]], [5], [0])
    tab = st["h32"][4:20].view(2, 8).tolist()
    assert tab == [[1, 3, 2, 4, 8, 8, 8, 8], [8] * 8] and st["h32"][20:].tolist() == [0, 2]


def test_token_ids_are_checked_on_the_host():
    from pmetal_b200.models.generation import Generator
    m = build_model(MODELS["ones"], torch.float32, "cpu")
    g = Generator(m, cache=m.new_cache(4, max_seqs=2))
    s = g.new_seq()
    for bad in ([40], [-1]):
        with pytest.raises(ValueError, match="token ids"):
            g.step([s], [bad])
    with pytest.raises(ValueError, match="at least one"):
        g.step([s], [[]])
    with pytest.raises(ValueError, match="wanted place"):
        g.step([s], [[1, 2]], [[2]])
    assert g.cache.length(s) == 0


def test_engine_admits_by_state_slots_and_presets_build():
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    m = build_model(MODELS["ones"], torch.float32, "cpu")
    e = ContinuousBatchEngine(m, max_slots=3, num_blocks=64)
    assert e.cache.max_seqs == 3 and e.prefix is None and e.mixed
    for _ in range(5):
        e.submit(Request([1, 2, 3]))
    e._admit()
    assert len(e.slots) == 3 and not e.cache.can_admit()
    with pytest.raises(ValueError, match="token ids"):
        e.submit(Request([1, 99]))
    for p in PRESETS.values():
        HybridDecoderLM(HybridArgs.from_dict(p), torch.bfloat16, "meta")
    a, args, d = load_pretrained("random:duvivik-tiny", torch.float32)
    assert d is None and args.model_type == "duvivik" and float(a.embed_tokens.abs().sum()) > 0


def _planted(monkeypatch, what):
    if what == "far key":                                   # the first page is not seen from beyond 100 positions
        real = O.latent_attention

        def cut(h, p, pre, m, c, kr):
            out = real(h, p, pre, m, c, kr)
            tail = real(h[64:], p, pre, m, c[64:], kr[64:]) if h.shape[0] > 100 else None
            return out if tail is None else torch.cat([out[:100], tail[36:]])
        monkeypatch.setattr(O, "latent_attention", cut)
    elif what == "rotation":                                # half-split pairs instead of neighbours
        real = O.rotate_pairs

        def halves(x, base, pos=None):
            d = x.shape[-1]
            ix = torch.arange(d).view(2, d // 2).t().reshape(-1)
            return real(x[..., ix], base, pos)[..., torch.argsort(ix)]
        monkeypatch.setattr(O, "rotate_pairs", halves)
    elif what == "state":                                   # state lost at a boundary of 64 tokens
        real = O.ssd_recurrence

        def lost(x, B, C, dt, A_log, D, S=None):
            parts = [real(x[i:i + 64], B[i:i + 64], C[i:i + 64], dt[i:i + 64], A_log, D)[0] for i in range(0, x.shape[0], 64)]
            return torch.cat(parts), None
        monkeypatch.setattr(O, "ssd_recurrence", lost)
    elif what == "taps":                                    # inputs before a portion are forgotten
        real = O.causal_conv
        monkeypatch.setattr(O, "causal_conv", lambda x, w, b: torch.cat([real(x[:64], w, b), real(x[64:], w, b)]))
    elif what == "gate":                                    # norm before the gate
        monkeypatch.setattr(O, "gated_group_norm", lambda y, z, w, n, eps: torch.cat(
            [O.rms(c, eps) for c in y.chunk(n, -1)], -1) * w * z * torch.sigmoid(z))
    elif what == "norm parts":
        real = O.gated_group_norm
        monkeypatch.setattr(O, "gated_group_norm", lambda y, z, w, n, eps: real(y, z, w, 1, eps))
    elif what == "limit":
        real = O.clamped_glu
        monkeypatch.setattr(O, "clamped_glu", lambda h, p, pre, limit: real(h, p, pre, 1e9))


@pytest.mark.parametrize("what", ["far key", "rotation", "state", "taps", "gate", "norm parts", "limit"])
def test_faults_show_in_the_test_model(monkeypatch, what):
    """The model the comparisons below use makes each of these mistakes visible well above the bf16 tolerance."""
    toks = tokens(150, 101, 5)
    want, tol = oracle("mixed", toks), bound("mixed", toks, torch.bfloat16)
    cfg = MODELS["mixed"]
    sd = {k: v.double() for k, v in random_weights(cfg).items()}
    _planted(monkeypatch, what)
    bad = O.forward(toks, sd, cfg)[0]
    assert err(bad[101:], want[101:]) > 2 * tol


# ------------------------------------------------------------------------------------------- kernels and mixers
@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 42, 1000, 2560])
def test_stream_kernels(dtype, width):
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(width)
    table = torch.randn(33, width, generator=g).to(dtype)
    ids = torch.tensor([0, 32, 5, 5, 17])
    xf, xc = nat.embed_scale(ids.cuda(), table.cuda(), 0.37)
    want = table.float()[ids] * 0.37
    torch.testing.assert_close(xf.cpu(), want, rtol=1e-6, atol=0)
    assert torch.equal(xc.cpu(), xf.cpu().to(dtype))
    x = torch.randn(9, width, generator=g) * 3 + 5          # a mean far from zero: the variance takes deviations
    ybuf = torch.randn(9, width + 8, generator=g).to(dtype)
    w, b, yb = torch.randn(3, width, generator=g).unbind(0)
    y = ybuf.cuda()[:, :width]
    of, oc = nat.post_layernorm(x.cuda(), y, w.cuda(), b.cuda(), 1e-4, 1.7, bias=yb.cuda())
    want = O.layer_norm(1.7 * x.double() + ybuf[:, :width].double() + yb.double(), w.double(), b.double(), 1e-4)
    torch.testing.assert_close(of.cpu().double(), want, rtol=2e-5, atol=2e-5)
    assert oc.dtype == dtype and torch.equal(oc.cpu(), of.cpu().to(dtype))
    rows = torch.tensor([8, 0, 3])
    none, oc = nat.post_layernorm(x.cuda(), None, w.cuda(), b.cuda(), 1e-4, rows=rows.cuda(), want_stream=False, dtype=dtype)
    want = O.layer_norm(x.double()[rows], w.double(), b.double(), 1e-4)
    torch.testing.assert_close(oc.cpu().double(), want, rtol=1e-2 if dtype == torch.bfloat16 else 2e-5, atol=1e-2 if dtype == torch.bfloat16 else 2e-5)


def _glu_weights(width, ff, gen, dtype):
    sh = {"gate": (ff, width), "gate.b": (ff,), "up": (ff, width), "up.b": (ff,), "down": (width, ff), "down.b": (width,)}
    return {"m." + k: (torch.randn(s, generator=gen) * (1.0 if len(s) == 1 else 2.0 * s[1] ** -0.5)).to(torch.bfloat16).double()
            for k, s in sh.items()}


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,limit", [(64, 96, 1.3), (42, 33, 0.5), (128, 256, 7.0)])
def test_clamped_feed_forward(dtype, width, ff, limit):
    from pmetal_b200.models.hybrid_decoder import ClampedMLP
    g = torch.Generator().manual_seed(ff)
    p = _glu_weights(width, ff, g, dtype)
    mod = ClampedMLP({"ff": ff, "limit": limit}, width, dtype, "cuda")
    with torch.no_grad():
        for name, _, put, _ in mod.named_weights():
            put(p["m." + name])
    for n in (1, 7, 16, 40):                                 # mat-vec epilogue and GEMM + gate kernel
        h = torch.randn(n, width, generator=g).to(dtype)
        got = mod(h.cuda())[:, :width].float() + mod.b_down
        run = lambda: O.clamped_glu(h.double(), p, "m.", limit)      # noqa: E731
        assert err(got, run()) < (bf16_bound(run, run()) if dtype == torch.bfloat16 else 1e-5)


@gpu
def test_rotation_table_far_positions():
    from pmetal_b200.models.mixers import RotationFreqs
    from pmetal_b200.ops import native as nat
    for base, dims in ((10000.0, 32), (1e6, 2), (37.5, 10)):
        pos = [0, 1, 63, 64, 4095, 131071, 1999999]
        cs, sn = nat.rope_table_f64(torch.tensor(pos, dtype=torch.int32).cuda(), RotationFreqs().get(base, dims, "cuda"))
        x = torch.zeros(len(pos), dims, dtype=torch.float64)
        x[:, 0::2] = 1.0                                     # (1, 0) turned: cos and sin
        want = O.rotate_pairs(x, base, pos)
        torch.testing.assert_close(cs.cpu().double(), want[:, 0::2], rtol=0, atol=3e-7)
        torch.testing.assert_close(sn.cpu().double(), want[:, 1::2], rtol=0, atol=3e-7)


def _mixer(m, width, dtype, seed, gain=1.0):
    """A mixer alone with a cache: returns (module, oracle weights 'w.', cache factory)."""
    cfg = config([(m, None, 0)], width=width)
    sd = random_weights(cfg, seed)
    model = build_model(cfg, dtype, "cuda")
    model.load_hf_state_dict(sd)
    return model.layers[0].mixer, {k: v.double() for k, v in sd.items()}, model


def _run_mixer(mix, model, h, sizes, order=None):
    """h [T, width] through the mixer in portions; the sequence sits in the second slot and in shuffled pages."""
    from pmetal_b200.models.mixers import StepContext
    cache = model.new_cache(40, max_seqs=3)
    cache.free = [b for b in range(0, 40, 2)] + [b for b in range(1, 40, 2)]
    cache.add_sequence(0)
    cache.add_sequence(1)
    for t in list(cache.pages.values()) + [t for d in cache.slots.values() for t in d.values()]:
        t.fill_(7.0)                                         # what an earlier owner may have left
    for t in cache.pages.values():
        t[..., sum(mix.dims[i] for i in (4, 2)):] = 0        # pad columns are never written
    out, at, k = [], 0, 0
    while at < h.shape[0]:
        n = min(sizes[min(k, len(sizes) - 1)], h.shape[0] - at)
        meta = cache.prepare([1], [n])
        out.append(mix(h[at:at + n].contiguous(), cache, StepContext(meta, model._freqs))[:, :h.shape[1]])
        at, k = at + n, k + 1
    return torch.cat(out)


PORTIONS = [[400], [1], [2], [3, 17, 64, 1, 1, 65, 2, 30], [16], [17], [63, 1, 64, 2], [100, 1, 1, 1, 40]]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [ssm(6, 20, 16, 3, 4, 2), ssm(4, 32, 48, 1, 3, 4), ssm(3, 7, 10, 3, 5, 3), ssm(1, 16, 16, 1, 1, 1),
                               ssm(2, 64, 128, 2, 4, 1), ssm(2, 40, 144, 1, 2, 2), ssm(4, 96, 64, 2, 4, 2), ssm(2, 2, 1, 1, 4, 1)],
                         ids=lambda m: f"h{m['heads']}p{m['vdim']}n{m['state']}k{m['conv']}")
def test_mamba2_mixer(dtype, m):
    mix, p, model = _mixer(m, 48, dtype, 1)
    h = torch.randn(200, 48, generator=torch.Generator().manual_seed(2)).to(dtype)
    run = lambda: O.mamba2(h.double(), p, "l0.mix.", m, 1e-5)      # noqa: E731
    want = run()
    tol = bf16_bound(run, want) if dtype == torch.bfloat16 else FP32
    for sizes in PORTIONS:
        got = _run_mixer(mix, model, h.cuda(), sizes)
        assert err(got, want) < tol, sizes


@gpu
def test_chunked_recurrence_keeps_fp32_factors():
    """Fast decays next to slow ones and states much larger than their updates: the block kernel and the scan agree far
    below bf16 rounding of the state."""
    from pmetal_b200.ops import native as nat
    H, P, N, G, taps = 4, 32, 64, 2, 4
    g = torch.Generator().manual_seed(0)
    T, conv = 330, H * P + 2 * G * N
    u = torch.randn(T, H * P + conv + H, generator=g).to(torch.bfloat16).cuda()
    cw, cb = (torch.randn(taps, conv, generator=g) * 0.5).cuda(), (torch.randn(conv, generator=g) * 0.1).cuda()
    dtb, al, D = torch.tensor([-6.0, -3.0, 0.0, 2.0]).cuda(), torch.tensor([-5.0, 0.0, 1.0, 2.5]).cuda(), torch.ones(H).cuda()
    out = []
    for fn in (nat.ssm_scan, nat.ssm_chunk):
        c = StateCache([CacheSpec(slots={"conv": ((taps, conv), None), "state": ((H, N, P), torch.float32)})], 16, 2,
                       torch.bfloat16, "cuda")
        c.add_sequence(0)
        c.slots[0]["state"].normal_(generator=torch.Generator(device="cuda").manual_seed(1))
        c.slots[0]["state"] *= 30
        c.slots[0]["conv"].normal_(generator=torch.Generator(device="cuda").manual_seed(2))
        c.prepare([0], [9])                                  # the state counts: the portion starts at position 9
        group, _ = split_groups(c.prepare([0], [T]), 1 << 30)
        y = torch.zeros(T, H * P, dtype=torch.bfloat16, device="cuda")
        fn(u, cw, cb, dtb, al, D, c.slots[0]["conv"], c.slots[0]["state"], group, (H, P, N, G, taps), y)
        out.append((y.float(), c.slots[0]["state"][c.slot_of[0]].clone()))
    (ya, sa), (yb, sb) = out
    assert float((ya - yb).norm() / ya.norm()) < 6e-3        # bf16 activations of the convolution, bf16 outputs
    for h in range(H):
        assert float((sa[h] - sb[h]).norm() / sa[h].norm()) < 4e-3
    assert float((sa[0] - sb[0]).norm() / sa[0].norm()) < 2e-4      # the slow head is dominated by the state it started from


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [attn(3, 16, 8, 24, 40), attn(5, 24, 8, 16, 96, base=1e6), attn(1, 11, 6, 3, 21), attn(20, 16, 16, 16, 128),
                               attn(2, 120, 32, 136, 72), attn(40, 8, 2, 8, 200), attn(2, 64, 64, 128, 512), attn(4, 96, 32, 64, 320)],
                         ids=lambda m: f"h{m['heads']}d{m['dim']}r{m['rot_dim']}v{m['vdim']}c{m['kv_rank']}")
def test_latent_attention_mixer(dtype, m):
    mix, p, model = _mixer(m, 48, dtype, 1)
    h = torch.randn(200, 48, generator=torch.Generator().manual_seed(4)).to(dtype)
    run = lambda: O.latent_attention(h.double(), p, "l0.mix.", m, *O.latent_kv(h.double(), p, "l0.mix.", m, 1e-5))      # noqa: E731
    want = run()
    tol = bf16_bound(run, want) if dtype == torch.bfloat16 else FP32
    for sizes in PORTIONS:
        got = _run_mixer(mix, model, h.cuda(), sizes)
        assert err(got, want) < tol, sizes


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_far_key_stands_out(dtype):
    """A query that scores one key far above all others reads that key's value, wherever it lies: the first tokens, both
    sides of page borders, the token itself; in prompts (expanded keys) and in decoding (latent space, split keys)."""
    W, T, probes = 64, 900, [0, 1, 63, 64, 127, 128, 500, 831, 832]
    m = attn(2, 32, 2, 32, 64, scale=1.0)
    mix, _, model = _mixer(m, W, dtype, 0)
    g = torch.Generator().manual_seed(1)
    # latents = the token vector itself; head keys / values = halves of it; rotated part switched off
    eye = torch.eye(W)
    with torch.no_grad():
        mix.w_q.zero_()
        mix.w_q[0:32], mix.w_q[34:66] = eye[:32].to(dtype), eye[32:].to(dtype)
        mix.w_q[mix.n_q:mix.n_q + 64] = eye.to(dtype)
        mix.norm_w.fill_(1.0)
        mix.w_ukv[:64], mix.w_ukv[64:128] = eye.to(dtype), eye.to(dtype)
        mix.w_o[:64] = eye.to(dtype)
    base = torch.randn(T, W, generator=g).sign()             # unit entries: rms 1
    from pmetal_b200.models.mixers import StepContext
    cache = model.new_cache(32, max_seqs=1)
    cache.add_sequence(0)
    h = base.to(dtype).cuda()
    mix(h, cache, StepContext(cache.prepare([0], [T]), model._freqs))
    for n in (1, 24):
        for at in range(0, len(probes), n):
            ps = probes[at:at + n]
            q = torch.stack([base[p] * 4.0 for p in ps] + [base[0] * 4.0] * (n - len(ps)))
            got = mix(q.to(dtype).cuda(), cache, StepContext(cache.prepare([0], [n]), model._freqs)).float().cpu()
            for i, p in enumerate(ps):
                assert torch.allclose(got[i], base[p], atol=2e-2), (n, p)


# ------------------------------------------------------------------------------------------- whole models
@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(MODELS))
def test_model_whole_portions_and_decoding(name, dtype):
    cfg, _, m = built(name, dtype)
    toks = tokens(150, cfg["vocab"], 5)
    want, tol = oracle(name, toks), bound(name, toks, dtype)
    assert err(m(torch.tensor(toks, device="cuda")), want) < tol
    docs = torch.tensor(toks[:70] + toks, device="cuda")                                  # two documents in one stream
    got = m(docs, cu_seqlens=torch.tensor([0, 70, 220], device="cuda"))
    assert err(got[:70], want[:70]) < tol and err(got[70:], want) < tol
    for sizes in ([150], [130, 1], [2], [1], [64, 1, 1, 63, 3], [5, 20, 70, 2, 1, 1]):
        gen = generator(m)
        got = feed(gen, gen.new_seq(), toks, sizes)
        assert err(got, want) < tol, sizes
        assert gen.cache.length(0) == 150


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mixed_batches_with_recycled_pages_and_slots(dtype):
    """Four live requests of unequal lengths, portions beside single tokens, pauses, ends and new requests in used pages and
    slots (overwritten with large values in between); every logit equals the request's own."""
    cfg, _, m = built("mixed", dtype)
    lens = {"a": 150, "b": 40, "c": 97, "d": 130, "e": 64, "f": 21, "g": 3}
    req = {k: tokens(n, cfg["vocab"], 10 + i) for i, (k, n) in enumerate(lens.items())}
    plan = [  # one dict per step: request -> number of tokens
        {"a": 2, "b": 30, "c": 1}, {"a": 70, "b": 1, "d": 64}, {"a": 1, "c": 60, "d": 1}, {"b": 1, "d": 1}, {"a": 20, "b": 8, "c": 2, "d": 1},
        {"a": 1, "c": 1, "d": 1, "e": 63}, {"a": 40, "d": 5, "e": 1}, {"a": 15, "c": 33, "d": 57, "f": 18}, {"a": 1, "f": 1}, {"f": 2, "g": 2},
        {"g": 1}]
    gen = generator(m, blocks=9, max_seqs=4)
    seq, at, got = {}, {k: 0 for k in req}, {k: [] for k in req}
    for step in plan:
        for k in step:
            if k not in seq:
                seq[k] = gen.new_seq()
        ks = list(step)
        out = gen.step([seq[k] for k in ks], [req[k][at[k]:at[k] + step[k]] for k in ks], [list(range(step[k])) for k in ks])
        out, o = out.float().cpu(), 0
        for k in ks:
            got[k].append(out[o:o + step[k]])
            o += step[k]
            at[k] += step[k]
            if at[k] == len(req[k]):
                c, blocks, slot = gen.cache, gen.cache.seqs[seq[k]].blocks, gen.cache.slot_of[seq[k]]
                c.free_sequence(seq[k])
                for t in c.pages.values():
                    t[blocks] = 50.0
                for mix in (l.mixer for l in m.layers if not l.mixer.cache_spec().slots and l.mixer.own):
                    c.pages[mix.index][..., mix.dims[4] + mix.dims[2]:] = 0
                for d in c.slots.values():
                    for t in d.values():
                        t[slot] = 50.0
    assert all(at[k] == len(req[k]) for k in req) and gen.cache.num_free() == 9 and gen.cache.can_admit()
    for k in req:
        assert err(torch.cat(got[k]), oracle("mixed", req[k])) < bound("mixed", req[k], dtype), k


@gpu
@pytest.mark.parametrize("graphs", [True, False])
def test_long_decoding_in_a_batch(graphs):
    """Three requests decode 100 tokens together (fp32, captured steps or eager), crossing page borders at different steps."""
    cfg, _, m = built("mixed")
    gen = generator(m, blocks=16, max_seqs=3, cuda_graphs=graphs)
    req = [tokens(n, cfg["vocab"], 20 + n) for n in (120, 163, 101)]
    seqs = [gen.new_seq() for _ in req]
    gen.prefill(seqs, [r[:len(r) - 100] for r in req])
    got = [gen.step(seqs, [[r[len(r) - 100 + i]] for r in req]).cpu() for i in range(100)]
    assert (gen._graphed is not None) == graphs
    for j, r in enumerate(req):
        assert err(torch.stack([g[j] for g in got]), oracle("mixed", r)[-100:]) < FP32


def _greedy(name, prompt, n):
    cfg = MODELS[name]
    sd = {k: v.double() for k, v in random_weights(cfg).items()}
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(O.forward(seq, sd, cfg)[0][-1].argmax()))
    return seq[len(prompt):]


@gpu
def test_greedy_generation_through_the_engine():
    """More requests than slots; prompts longer than a prefill portion run beside decoding slots in one batch."""
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    cfg, _, m = built("ones")
    prompts = [tokens(n, cfg["vocab"], 30 + n) for n in (5, 70, 1, 33, 90)]
    want = [_greedy("ones", p, 8) for p in prompts]
    e = ContinuousBatchEngine(m, max_slots=2, num_blocks=8, prefill_chunk=31)
    mixed = []
    step = e.gen.step
    e.gen.step = lambda s, t, w=None: mixed.append([len(x) for x in t]) or step(s, t, w)
    reqs = [e.submit(Request(p, SamplingParams.greedy(8))) for p in prompts]
    while not all(r.done.is_set() for r in reqs):
        assert e.tick()
    assert [r.output for r in reqs] == want and any(len(x) == 2 and max(x) > 1 for x in mixed)
    assert e.cache.num_free() == 8 and len(e.cache.free_slots) == 2
    from pmetal_b200.models.generation import Generator
    g = Generator(m, cache=m.new_cache(16, max_seqs=6))
    res = g.generate(prompts[:2], SamplingParams.greedy(8), num_return_sequences=3)      # forks share pages, copy states
    assert res.tokens == [want[0]] * 3 + [want[1]] * 3
    assert list(g.stream(prompts[3], SamplingParams.greedy(8))) == want[3]
    assert len(g.cache.free_slots) == 6 and g.cache.num_free() == 16


@gpu
def test_attention_only_stack_shares_prompt_prefixes():
    """Without recurrent layers prompts may be parked and cut at block borders: a second request forks the cached pages."""
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine
    cfg = config([(attn(2, 16, 8, 16, 32), 32, 1.0), (attn(3, 16, 8, 8, 32, kv_from=0), None, 0)], width=32, vocab=60)
    sd = random_weights(cfg, 2)
    m = build_model(cfg, torch.float32, "cuda")
    m.load_hf_state_dict(sd)
    e = ContinuousBatchEngine(m, max_slots=2, num_blocks=24)
    p = tokens(150, 60, 9)
    a = e.generate(p, SamplingParams.greedy(4))
    b = e.generate(p[:140] + [1, 2, 3], SamplingParams.greedy(4))
    ref = ContinuousBatchEngine(m, max_slots=2, num_blocks=24, prefix_cache=False)
    assert e.stats.prefix_hits == 1 and b.cached_tokens == 128
    assert a.output == ref.generate(p, SamplingParams.greedy(4)).output
    assert b.output == ref.generate(p[:140] + [1, 2, 3], SamplingParams.greedy(4)).output


@gpu
def test_sampled_requests_and_background_thread():
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine
    _, _, m = built("odd", torch.bfloat16)
    e = ContinuousBatchEngine(m, max_slots=4, num_blocks=16)
    e.start()
    try:
        a = e.generate([3, 5, 7], SamplingParams(temperature=0.8, top_p=0.9, max_tokens=12, seed=4), want_logprobs=True)
        b = e.generate([3, 5, 7], SamplingParams(temperature=1.0, repetition_penalty=1.3, max_tokens=12, seed=4))
    finally:
        e.shutdown()
    assert len(a.output) == 12 and len(a.logprobs) == 12 and all(0 <= t < 77 for t in a.output + b.output)


@gpu
def test_command_line(tmp_path, capsys):
    from pmetal_b200.cli.main import main
    cfg = copy.deepcopy(PRESETS["duvivik-tiny"])
    m = build_model(cfg, torch.float32, "cpu").init_weights(0.05, 3)
    save_pretrained(m, str(tmp_path))
    assert main(["infer", "-m", str(tmp_path), "-p", "hello", "--greedy", "--max-tokens", "5", "--json", "--kv-blocks", "16"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["generated_tokens"] == 5 and out["prompt_tokens"] == 5
    assert main(["infer", "-m", "random:duvivik-tiny", "-p", "hi", "--profile-layers", "--json"]) == 0
    assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["layers"]) == 4
    data = tmp_path / "d.jsonl"
    data.write_text('{"text": "some words"}\n{"text": "and a few more"}\n')
    assert main(["eval", "-m", str(tmp_path), "-d", str(data)]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["perplexity"] > 1
    with pytest.raises(SystemExit, match="--lora"):
        main(["infer", "-m", str(tmp_path), "-p", "x", "-l", str(tmp_path)])


@gpu
def test_http_server():
    from fastapi.testclient import TestClient

    from pmetal_b200.data.tokenizer import ByteTokenizer
    from pmetal_b200.serve.engine import ContinuousBatchEngine
    from pmetal_b200.serve.server import ServerState, create_app
    m, _, _ = load_pretrained("random:duvivik-tiny", torch.bfloat16, "cuda")
    eng = ContinuousBatchEngine(m, max_slots=2, num_blocks=16)
    eng.start()
    try:
        with TestClient(create_app(ServerState(eng, ByteTokenizer(), model_name="tiny"))) as c:
            r = c.post("/v1/completions", json={"model": "tiny", "prompt": "hi there", "max_tokens": 5, "temperature": 0}).json()
            assert r["usage"] == {"prompt_tokens": 8, "completion_tokens": 5, "total_tokens": 13}
            e = c.post("/v1/embeddings", json={"model": "tiny", "input": ["a", "some text"]}).json()
            assert len(e["data"]) == 2 and len(e["data"][0]["embedding"]) == m.cfg.hidden_size
    finally:
        eng.shutdown()


@gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(tmp_path, monkeypatch, capsys, dtype):
    """Steps on standard input, logits in files; the pool holds just what the live requests need."""
    import numpy as np
    from pmetal_b200.serve import trace
    cfg, _, _ = built("mixed")
    m = build_model(cfg, torch.bfloat16, "cpu")
    m.load_hf_state_dict(random_weights(cfg))
    save_pretrained(m, str(tmp_path / "m"))
    x, y, z = (tokens(n, cfg["vocab"], 50 + n) for n in (100, 30, 70))
    steps = [{"entries": [{"id": "x", "tokens": x[:99], "want": [0, 98]}], "end": []},
             {"entries": [{"id": "y", "tokens": y[:28], "want": []}, {"id": "x", "tokens": x[99:], "want": [0]}], "end": ["x"]},
             {"entries": [{"id": "y", "tokens": y[28:29], "want": []}], "end": []},
             {"entries": [{"id": "z", "tokens": z, "want": [69, 3]}, {"id": "y", "tokens": y[29:], "want": [0]}], "end": ["y", "z"]}]
    lines = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    monkeypatch.setattr(sys, "stdin", io.StringIO(lines))
    rc = trace.main(["--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path / "o"), "--max-tokens", "192"])
    assert rc == 0 and capsys.readouterr().out.split() == ["done", "0", "done", "1", "done", "2", "done", "3"]
    assert sorted(os.listdir(tmp_path / "o")) == ["0.f32", "1.f32", "3.f32"]
    load = lambda i: torch.from_numpy(np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])      # noqa: E731
    ox, oy, oz = oracle("mixed", x), oracle("mixed", y), oracle("mixed", z)
    tol = max(bound("mixed", t, getattr(torch, dtype)) for t in (x, y, z))
    assert err(load(0), ox[[0, 98]]) < tol and err(load(1), ox[[99]]) < tol
    assert err(load(3), torch.cat([oz[[69, 3]], oy[[29]]])) < tol


@gpu
def test_trace_replay_serves_the_dense_decoder_too():
    """The replay takes any model on the paged caches: portions, captured single steps and recycled blocks of the key / value
    cache against the model's own whole-sequence forward."""
    from pmetal_b200.models.config import ModelArgs
    from pmetal_b200.models.decoder import DecoderLM
    from pmetal_b200.serve.trace import TraceReplay
    cfg = ModelArgs(vocab_size=300, hidden_size=256, intermediate_size=320, num_hidden_layers=2, num_attention_heads=2,
                    num_key_value_heads=1, head_dim=128)
    m = DecoderLM(cfg).init_weights(0.05, 0).to("cuda").to(torch.bfloat16).eval()
    for p in m.parameters():
        p.requires_grad_(False)
    r = TraceReplay(m, 192)
    for seed in (1, 2):
        x, y = tokens(100, 300, seed), tokens(40, 300, 10 + seed)
        a = r.step([{"id": "x", "tokens": x[:70], "want": [0, 69]}], [])
        b = r.step([{"id": "y", "tokens": y[:39], "want": []}, {"id": "x", "tokens": x[70:99], "want": [28]}], [])
        assert r.step([{"id": "y", "tokens": y[39:], "want": []}], []) is None
        c = r.step([{"id": "x", "tokens": x[99:], "want": [0]}], ["x", "y"])
        want = m(torch.tensor(x, device="cuda")).double().cpu()
        assert err(torch.cat([a, b, c]), want[[0, 69, 98, 99]]) < 0.08
    assert r.gen.cache.num_free() == 3
