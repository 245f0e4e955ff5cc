"""Resevik on the hybrid decoder: kernels, mixers and experts against the plain statement in ``resevik_oracle.py``, then whole
models through the generator's step function, the paged state cache, the batching engine and the command line."""
import copy
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import resevik_oracle as O
from test_hybrid_decoder import FP32, PORTIONS, err, feed, generator, tokens

from pmetal_b200.models.architectures import build_model, family_of
from pmetal_b200.models.hybrid_decoder import PRESETS, HybridArgs, HybridDecoderLM
from pmetal_b200.models.kv_cache import BLOCK
from pmetal_b200.models.loader import load_pretrained, save_pretrained
from pmetal_b200.models.moe import WeightedInputExperts
from pmetal_b200.models.state_cache import CacheSpec, StateCache, split_groups

gpu = pytest.mark.gpu


# ------------------------------------------------------------------------------------------- models of the tests
def lightning(dim, vdim, decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def retention(dim, vdim, decay, rot=None, base=10000.0):
    return dict(lightning(dim, vdim, decay), rot={"base": base, "dims": dim if rot is None else rot})


def attn(heads, kv, dim, window, rot, base=10000.0, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "mask": {"size": window}, "rot": {"base": base, "dims": rot},
            "scale": scale or 2.5 * dim ** -0.5}


def kind(m):
    return "attention" if "mask" in m else ("retention" if "rot" in m else "lightning")


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, loop=None, width=48, vocab=101, scale=1.0, eps=1e-5):
    """layers: (mixer, feed-forward or None)."""
    d = {"architecture": "Resevik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
         "layers": [{"type": kind(m), "mixer": m, "mlp": f} for m, f in layers]}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


MODELS = {
    # every mixer, two windows, layers before, in and behind the loop, one without feed-forward, partial and whole rotations
    "mixed": config([(lightning(16, 24, [0.4, 0.9, 0.995]), moe(40, 7, 3)), (retention(24, 40, [0.97, 0.999], 16), moe(24, 4, 1)),
                     (attn(6, 2, 20, 40, 12), moe(48, 5, 2)), (lightning(32, 8, [0.8, 0.99]), None),
                     (attn(3, 3, 32, 70, 32, base=500.0), moe(16, 6, 6)), (retention(16, 16, [0.9]), moe(32, 3, 2))], (1, 4, 3)),
    # sizes that are not multiples of what the fast kernels copy at a time, no loop
    "odd": config([(lightning(10, 7, [0.7, 0.99, 0.3]), moe(33, 5, 1)), (retention(14, 5, [0.98], 6, 37.0), moe(21, 3, 2)),
                   (attn(3, 1, 11, 9, 6), None), (retention(6, 9, [0.5, 0.995]), None), (attn(2, 2, 26, 33, 0), moe(10, 2, 1))],
                  width=42, vocab=77, scale=1.9, eps=1e-3),
    # everything that may be one
    "ones": config([(lightning(1, 1, [1.0]), moe(1, 1, 1)), (attn(1, 1, 8, 1, 2), moe(8, 3, 1)), (retention(2, 1, [1.0]), None),
                    (retention(2, 4, [0.0, 0.6]), moe(8, 2, 1))], (0, 1, 1), width=32, vocab=40),
    # heads wider than one tile, than the block recurrence and than the tensor-core attention take; the whole stack loops
    "wide": config([(lightning(144, 136, [0.9, 0.999]), moe(64, 40, 4)), (retention(264, 72, [0.99]), None), (attn(2, 1, 264, 100, 64), None),
                    (attn(4, 2, 192, 65, 192), None), (attn(10, 1, 128, 64, 32), moe(72, 9, 2)), (retention(128, 40, [0.95, 0.998], 96), None)],
                   (0, 6, 2), width=64, vocab=90),
    # attention alone: the pages are all there is, the window decides when they go back to the pool
    "pages": config([(attn(4, 2, 16, 50, 8), moe(24, 4, 2)), (attn(2, 2, 24, 30, 24), None)], (0, 2, 2), width=32, vocab=60),
}
CENTRES = 4


def random_weights(cfg, seed=0):
    """bf16-representable weights. Token vectors lie around a few centres and the routers tell the centres apart, so that
    rounding does not change which experts are chosen; sublayers add little to each sum, so that this holds in every layer."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    centres = torch.linalg.qr(torch.randn(W, CENTRES, generator=g))[0].t() * W ** 0.5
    sd = {}
    for name, shape, _, _ in HybridDecoderLM(HybridArgs.from_dict(cfg), device="meta").named_weights():
        leaf = name.rsplit(".", 1)[-1]
        n = lambda s=1.0: torch.randn(shape, generator=g) * s      # noqa: E731
        if leaf == "router":
            top = cfg["layers"][int(name[1:].split(".")[0])]["mlp"]["router"]["top"]
            lv = torch.full((shape[0], CENTRES), -1.5)
            for c in range(CENTRES):
                lv[torch.randperm(shape[0], generator=g)[:top], c] = 1.5
            t = lv @ centres / W + n(0.05 * W ** -0.5)
        elif leaf in ("norm", "norm1"):
            t = torch.rand(shape, generator=g) * 0.4 + 0.8
        elif leaf == "embed":
            t = (centres[torch.arange(shape[0]) % CENTRES] + n(0.5)) / cfg["embedding"]["scale"] * 2
        elif leaf in ("o", "down"):
            t = n(0.5 * shape[1] ** -0.5)
        else:
            t = n(shape[1] ** -0.5)
        sd[name] = t.to(torch.bfloat16)
    return sd


_CACHE = {}


def cached(key, make):
    if key not in _CACHE:
        _CACHE[key] = make()
    return _CACHE[key]


def weights64(name):
    return cached(("w", name), lambda: {k: v.double() for k, v in random_weights(MODELS[name]).items()})


def built(name, dtype=torch.float32, device="cuda"):
    def make():
        m = build_model(MODELS[name], dtype, device)
        assert m.load_hf_state_dict(random_weights(MODELS[name])) == []
        return m.eval()
    return MODELS[name], cached(("m", name, dtype, device), make)


def oracle(name, toks):
    return cached(("o", name, tuple(toks)), lambda: O.forward(list(toks), weights64(name), MODELS[name])[0])


def bf16_bound(run, want):
    """Twice what rounding the oracle's own projections and activations to bf16 does to it in the worst row, plus a little."""
    with O.rounding():
        return 2 * err(run(), want) + 5e-3


def bound(name, toks, dtype):
    if dtype == torch.float32:
        return FP32
    return cached(("b", name, tuple(toks)),
                  lambda: bf16_bound(lambda: O.forward(list(toks), weights64(name), MODELS[name])[0], oracle(name, toks)))


# ------------------------------------------------------------------------------------------- host side (no GPU)
def test_registry_and_configuration():
    cfg = MODELS["mixed"]
    assert family_of(cfg) == "hybrid" and family_of({"model_type": "resevik"}) == "hybrid"
    a = HybridArgs.from_dict(cfg)
    assert (a.vocab_size, a.hidden_size, a.num_hidden_layers, a.norm_eps, a.loop) == (101, 48, 6, 1e-5, (1, 4, 3))
    assert a.runs == O.runs(cfg) and [i for i, _ in a.runs] == [0] + [1, 2, 3] * 3 + [4, 5]
    assert [n for n, (_, again) in enumerate(a.runs) if again] == [4, 7]
    assert HybridArgs.from_dict(dict(cfg, loop=None)).runs == [(i, False) for i in range(6)]
    assert a.to_hf_dict() == cfg and a.to_hf_dict() is not cfg
    m = build_model(cfg, torch.float32, "cpu")
    assert isinstance(m, HybridDecoderLM) and m.norm_b is None
    c = m.new_cache(4, max_seqs=2)                          # every layer run has pages or slots of its own
    assert sorted(c.pages) == [2, 5, 8, 10] and sorted(c.slots) == [0, 1, 3, 4, 6, 7, 9, 11]
    assert c.pages[2].shape == (5, BLOCK, 2 * 2 * 24) and c.slots[1]["state"].shape == (3, 2, 24, 40) and c.window == 70
    with pytest.raises(RuntimeError, match="CUDA"):
        m(torch.tensor([1, 2]))


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), "decays"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 1.5, 0.1]), "decays"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "rot"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "rot"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=4), "key/value"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=24), "vdim"),
    (lambda c: c["layers"][2]["mixer"].update(mask={"size": 0}), "mask"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0].update(type="mamba2"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "top"),
    (lambda c: c["loop"].update(stop=7), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].update(start=4), "loop"),
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
    with pytest.raises(KeyError, match="l0.mlp.e4.up"):
        m.load_hf_state_dict({k: v for k, v in sd.items() if k != "l0.mlp.e4.up"})
    with pytest.raises(ValueError, match="shape"):
        m.load_hf_state_dict(dict(sd, **{"l0.mix.norm": torch.zeros(4)}))


def test_windowed_pages_return_to_the_pool():
    """With a window on every layer that has pages, a page goes back once no later query can see it, not before."""
    specs = [CacheSpec(page_width=16, window=100), CacheSpec(slots={"state": ((4,), torch.float32)}), CacheSpec(page_width=8, window=30)]
    c = StateCache(specs, 8, 2, torch.float32, "cpu")
    assert c.window == 100 and not c.can_truncate
    assert StateCache([specs[0], CacheSpec(page_width=8)], 4, 1, torch.float32, "cpu").window == 0
    c.add_sequence(0)
    c.prepare([0], [163])                                   # the next query is position 163: it sees 64 .. 163
    assert c.num_free() == 5
    c.prepare([0], [1])
    assert c.num_free() == 6 and c.seqs[0].blocks[0] == -1 and c.seqs[0].blocks[1] >= 0
    m = c.prepare([0], [1])
    assert c.num_free() == 6 and m.block_table.tolist()[0][0] == 0 and m.block_table.tolist()[0][1:] == c.seqs[0].blocks[1:]
    assert c.can_admit()
    c.fork(0, 1)
    c.free_sequence(0)
    assert c.num_free() == 6
    c.free_sequence(1)
    assert c.num_free() == 8 and len(c.free_slots) == 2
    c.add_sequence(3)
    c.prepare([3], [162])
    c.prepare([3], [1])                                     # position 162 still sees position 63
    assert c.seqs[3].blocks[0] >= 0
    with pytest.raises(ValueError, match="window"):
        c.truncate(3, 100)


def test_engine_and_presets_build():
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    for name in ("ones", "pages"):
        m = build_model(MODELS[name], torch.float32, "cpu")
        e = ContinuousBatchEngine(m, max_slots=3, num_blocks=64)
        assert e.cache.max_seqs == 3 and e.prefix is None and e.mixed
        for _ in range(5):
            e.submit(Request([1, 2, 3]))
        e._admit()
        assert len(e.slots) == 3
    for p in ("resevik-tiny", "resevik-1b", "resevik-2b"):
        HybridDecoderLM(HybridArgs.from_dict(PRESETS[p]), torch.bfloat16, "meta")
    a, args, d = load_pretrained("random:resevik-tiny", torch.float32)
    assert d is None and args.model_type == "resevik" and float(a.embed_tokens.abs().sum()) > 0
    assert args.loop == (0, 3, 2)


def test_component_lists_name_existing_sources():
    from pmetal_b200 import build
    for stems in build.COMPONENTS.values():
        for s in stems:
            assert os.path.exists(os.path.join(build.CSRC, s + ".cu"))
    assert {"duvivik", "resevik"} <= set(build.COMPONENTS)


def _planted(monkeypatch, what):
    if what == "window":                                    # one token too many
        real = O.window_attention
        monkeypatch.setattr(O, "window_attention", lambda h, p, pre, m, eps: real(h, p, pre, dict(m, mask={"size": m["mask"]["size"] + 1}), eps))
        monkeypatch.setitem(O.MIXERS, "attention", O.window_attention)
    elif what == "values":                                  # normalised instead of projected keys as values
        real = O.linear
        real_attn = O.window_attention

        def attn_unit(h, p, pre, m, eps):
            T, G, D = h.shape[0], m["kv_heads"], m["dim"]

            def lin(x, w):
                y = real(x, w)
                return O.unit_rms(y.reshape(T, G, D), eps).reshape(T, G * D) if w is p[pre + "k"] else y
            monkeypatch.setattr(O, "linear", lin)
            out = real_attn(h, p, pre, m, eps)
            monkeypatch.setattr(O, "linear", real)
            return out
        monkeypatch.setitem(O.MIXERS, "attention", attn_unit)
    elif what == "rotation":                                # the other layout of pairs
        real = O.rotate
        monkeypatch.setattr(O, "rotate", lambda x, base, dims, layout: real(x, base, dims, {"half": "pairs", "pairs": "half"}[layout]))
    elif what == "state":                                   # state lost at a boundary of 64 tokens
        real = O.decayed_recurrence
        monkeypatch.setattr(O, "decayed_recurrence", lambda q, k, v, decay, S=None: (torch.cat(
            [real(q[i:i + 64], k[i:i + 64], v[i:i + 64], decay)[0] for i in range(0, q.shape[0], 64)]), None))
    elif what == "decay":                                   # the heads' decays in another order
        real = O.decayed_recurrence
        monkeypatch.setattr(O, "decayed_recurrence", lambda q, k, v, decay, S=None: real(q, k, v, decay[::-1]))
    elif what == "weight":                                  # the routing weight on the expert's output
        real = O.expert

        def mixture(h, p, pre, m):
            ids, wts = O.route(h, p[pre + "router"], m["router"]["top"])
            out = torch.zeros_like(h)
            for e in range(m["router"]["experts"]):
                for s in range(ids.shape[1]):
                    rows = (ids[:, s] == e).nonzero()[:, 0]
                    if rows.numel():
                        out[rows] = out[rows] + wts[rows, s, None] * real(h[rows], p, f"{pre}e{e}.")
            return out
        monkeypatch.setattr(O, "mixture", mixture)
    elif what == "top":                                     # one expert fewer
        real = O.route
        monkeypatch.setattr(O, "route", lambda h, w, top: tuple(t[:, :max(1, top - 1)] for t in real(h, w, top)))
    elif what == "loop":                                    # the embedding output is not added again
        real = O.runs
        monkeypatch.setattr(O, "runs", lambda cfg: [(i, False) for i, _ in real(cfg)])
    elif what == "passes":
        real = O.runs
        monkeypatch.setattr(O, "runs", lambda cfg: real(dict(cfg, loop=dict(cfg["loop"], times=cfg["loop"]["times"] - 1))))
    elif what == "head norm":                               # all heads of a retention layer normed together
        real = O.unit_rms
        monkeypatch.setattr(O, "unit_rms", lambda x, eps: real(x.flatten(1), eps).reshape(x.shape) if x.dim() == 3 else real(x, eps))
    elif what == "gate":
        monkeypatch.setattr(O, "silu", torch.sigmoid)


@pytest.mark.parametrize("what", ["window", "values", "rotation", "state", "decay", "weight", "top", "loop", "passes", "head norm", "gate"])
def test_faults_show_in_the_test_model(monkeypatch, what):
    """The model the comparisons below use makes each of these mistakes visible well above the bf16 tolerance."""
    toks = tokens(150, 101, 5)
    want, tol = oracle("mixed", toks), bound("mixed", toks, torch.bfloat16)
    _planted(monkeypatch, what)
    bad = O.forward(toks, weights64("mixed"), MODELS["mixed"])[0]
    assert err(bad[101:], want[101:]) > 2 * tol


def test_routers_of_the_test_models_decide_clearly(monkeypatch):
    """Rounding to bf16 does not change the chosen experts of any layer run."""
    real, gaps = O.route, []

    def watch(h, w, top):
        z = (h @ w.t()).sort(dim=-1, descending=True)[0]
        if top < z.shape[1]:
            gaps.append(float((z[:, top - 1] - z[:, top]).min()))
        return real(h, w, top)
    monkeypatch.setattr(O, "route", watch)
    for name, cfg in MODELS.items():
        O.forward(tokens(60, cfg["vocab"], 5), weights64(name), cfg)
    assert min(gaps) > 0.25


# ------------------------------------------------------------------------------------------- kernels and modules
@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 42, 1000, 2560])
def test_residual_sum_and_norm_kernel(dtype, width):
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    x, x0, w = r(9, width) * 3, r(9, width), r(width)
    ybuf, z = r(9, width + 8).to(dtype), r(20, width).to(dtype)
    inv = torch.randperm(20, generator=g)[:18].int()
    y = ybuf.cuda()[:, :width]
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)
    full = x.double() + ybuf[:, :width].double() + z.double()[inv.long()].view(9, 2, width).sum(1) + x0.double()
    xs = x.cuda()
    of, oc = nat.add_rmsnorm(xs, w.cuda(), 1e-3, y=y, z=z.cuda(), inv=inv.cuda(), k=2, x0=x0.cuda(), out=xs)
    assert of is xs and oc.dtype == dtype
    torch.testing.assert_close(of.cpu().double(), full, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(oc.cpu().double(), O.unit_rms(full, 1e-3) * w.double(), **tol)
    rows = torch.tensor([8, 0, 3])
    none, oc = nat.add_rmsnorm(x.cuda(), w.cuda(), 1e-3, y=y, rows=rows.cuda(), want_stream=False)
    want = O.unit_rms((x.double() + ybuf[:, :width].double())[rows], 1e-3) * w.double()
    assert none is None
    torch.testing.assert_close(oc.cpu().double(), want, **tol)
    _, oc = nat.add_rmsnorm(x.cuda(), w.cuda(), 1e-3, dtype=dtype, want_stream=False)
    torch.testing.assert_close(oc.cpu().double(), O.unit_rms(x.double(), 1e-3) * w.double(), **tol)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("silu", [True, False])
@pytest.mark.parametrize("n,parts,width", [(3, 4, 40), (3, 1, 512), (700, 5, 264), (700, 1, 1024), (2, 3, 7), (5, 1, 4104), (1, 1, 1)])
def test_norm_and_gate_kernel(dtype, silu, n, parts, width):
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(width + n)
    y, u = (torch.randn(n, c, generator=g).to(dtype) for c in (parts * width, parts * width + 24))
    w = torch.rand(parts * width, generator=g) + 0.5
    gate = u.double()[:, 8:8 + parts * width]
    gate = gate * torch.sigmoid(gate) if silu else torch.sigmoid(gate)
    unit = O.unit_rms(y.double().view(n, parts, width), 1e-4).view(n, -1)
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=3e-5, atol=1e-5)
    for wt in (w, None):
        got = nat.norm_gate(y.cuda(), u.cuda()[:, 8:8 + parts * width], None if wt is None else wt.cuda(), 1e-4, parts, silu)
        torch.testing.assert_close(got.cpu().double(), unit * gate * (1.0 if wt is None else wt.double()), **tol)


@gpu
@pytest.mark.parametrize("T,E,k", [(1, 1, 1), (5, 40, 4), (37, 7, 7), (700, 12, 2), (300, 64, 1), (1500, 3, 1)])
def test_sigmoid_routing(T, E, k):
    from pmetal_b200.ops import native as nat
    z = torch.randn(T, E + 3, generator=torch.Generator().manual_seed(T)) * 3
    s = torch.sigmoid(z[:, :E].double())
    want = s.sort(dim=-1, descending=True)
    for lg in (z.cuda()[:, :E], z.cuda()[:, :E].to(torch.bfloat16)):
        r = nat.moe_route(lg, k, False, score="sigmoid")
        ref = torch.sigmoid(lg.double().cpu()).sort(dim=-1, descending=True, stable=True)
        torch.testing.assert_close(r["topk_w"].cpu().double(), ref[0][:, :k], rtol=1e-5, atol=1e-6)
        assert torch.equal(r["topk_idx"].cpu().long(), ref[1][:, :k])
        perm, inv, off = r["perm"].cpu().long(), r["inv"].cpu().long(), r["offsets"].cpu()
        assert torch.equal(perm[inv], torch.arange(T * k)) and off[-1] == T * k
        e = r["topk_idx"].cpu().flatten()[perm]
        assert torch.equal(e, e.sort()[0]) and torch.equal(off.diff(), torch.bincount(e, minlength=E).int())
    soft = nat.moe_route(z.cuda()[:, :E], k, True)
    p = torch.softmax(z[:, :E].double(), -1).gather(1, want[1][:, :k])
    torch.testing.assert_close(soft["topk_w"].cpu().double(), p / p.sum(-1, keepdim=True), rtol=1e-4, atol=1e-6)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,experts,top", [(64, 96, 6, 2), (48, 8, 1, 1), (42, 33, 5, 3), (64, 24, 40, 4), (128, 256, 3, 1), (64, 72, 4, 4)])
def test_experts_with_weighted_inputs(dtype, width, ff, experts, top):
    """From one token to more rows than a tile per expert (narrow tiles, padded slabs, row kernel); experts without rows."""
    g = torch.Generator().manual_seed(ff)
    mod = WeightedInputExperts({"expert": {"ff": ff}, "router": {"experts": experts, "top": top}}, width, dtype, "cuda")
    p = {}
    with torch.no_grad():
        for name, shape, put, get in mod.named_weights():
            p["m." + name] = (torch.randn(shape, generator=g) * (1.5 if name == "router" else 1.8) * shape[1] ** -0.5).to(torch.bfloat16)
            put(p["m." + name])
            assert torch.equal(get().cpu().to(torch.bfloat16), p["m." + name])
    p = {n: t.double() for n, t in p.items()}
    for n in (1, 2, 7, 16, 40, 333, 900):
        h = torch.randn(4 * n, width, generator=g).to(dtype)
        z = (h.double() @ p["m.router"].t()).sort(-1, descending=True)[0]     # tokens whose choice is no close call
        clear = (z[:, top - 1] - z[:, top] > 0.02) if top < experts else torch.ones(4 * n, dtype=torch.bool)
        h = h[clear][:n]
        rows, inv, k = mod(h.cuda())
        got = rows.double().cpu()[inv.cpu().long()].view(h.shape[0], k, width).sum(1)
        run = lambda: O.mixture(h.double(), p, "m.", {"router": {"experts": experts, "top": top}})      # noqa: E731
        assert err(got, run()) < (bf16_bound(run, run()) if dtype == torch.bfloat16 else 1e-5), n
    from pmetal_b200.ops import native as nat
    nat.check_status()


def _mixer(m, width, dtype, seed):
    cfg = config([(m, None)], width=width)
    sd = random_weights(cfg, seed)
    model = build_model(cfg, dtype, "cuda")
    model.load_hf_state_dict(sd)
    return model.layers[0].mixer, {k: v.double() for k, v in sd.items()}, model


def _run_mixer(mix, model, h, sizes):
    """h [T, width] through the mixer in portions; the sequence sits in the second slot and in shuffled pages, which hold what
    an earlier owner may have left."""
    from pmetal_b200.models.mixers import StepContext
    cache = model.new_cache(40, max_seqs=3)
    cache.free = [b for b in range(0, 40, 2)] + [b for b in range(1, 40, 2)]
    cache.add_sequence(0)
    cache.add_sequence(1)
    for t in list(cache.pages.values()) + [t for d in cache.slots.values() for t in d.values()]:
        t.fill_(7.0)
    out, at, k = [], 0, 0
    while at < h.shape[0]:
        n = min(sizes[min(k, len(sizes) - 1)], h.shape[0] - at)
        meta = cache.prepare([1], [n])
        out.append(mix(h[at:at + n].contiguous(), cache, StepContext(meta, model._freqs), 0)[:, :h.shape[1]])
        at, k = at + n, k + 1
    return torch.cat(out)


def _id(m):
    return f"{kind(m)[:4]}-h{m['heads']}d{m['dim']}v{m['vdim']}" + (f"w{m['mask']['size']}r{m['rot']['dims']}" if "mask" in m else "")


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [
    lightning(16, 24, [0.4, 0.9, 0.995]), lightning(10, 7, [0.7, 0.99, 0.3]), lightning(1, 3, [1.0]), lightning(128, 64, [0.999, 0.6]),
    lightning(144, 136, [0.97]), lightning(256, 40, [0.99]), lightning(264, 8, [0.99, 0.0]), lightning(8, 100, [0.999] * 5),
    retention(24, 40, [0.97, 0.999], 16), retention(14, 5, [0.98], 6, 37.0), retention(2, 1, [1.0]), retention(128, 96, [0.95, 0.998]),
    retention(64, 32, [0.9, 0.0, 1.0], 48, 1e6), retention(200, 64, [0.995], 128), retention(272, 16, [0.99]), retention(32, 16, [0.9], 0)], ids=_id)
def test_linear_attention_mixers(dtype, m):
    mix, p, model = _mixer(m, 48, dtype, 1)
    h = torch.randn(200, 48, generator=torch.Generator().manual_seed(2)).to(dtype)
    run = lambda: O.MIXERS[kind(m)](h.double(), p, "l0.mix.", m, 1e-5)      # noqa: E731
    want = run()
    # a key of one channel leaves states and outputs near zero that the norm blows up: what fp32 does to the oracle counts
    single = O.MIXERS[kind(m)](h.float(), {k: v.float() for k, v in p.items()}, "l0.mix.", m, 1e-5)
    tol = bf16_bound(run, want) if dtype == torch.bfloat16 else max(FP32, 6 * err(single, want))
    for sizes in PORTIONS:
        assert err(_run_mixer(mix, model, h.cuda(), sizes), want) < tol, sizes


@gpu
def test_block_recurrence_keeps_fp32_factors():
    """Rotated queries and keys are fp32 values: block kernel and scan agree far below bf16 rounding of either, also on a state
    much larger than its updates, over several parallel segments."""
    from pmetal_b200.ops import native as nat
    H, N, P, T = 3, 64, 40, 1500
    g = torch.Generator().manual_seed(0)
    u = torch.randn(T, H * (2 * N + P), generator=g).to(torch.bfloat16).cuda()
    ang = torch.rand(T, N // 2, generator=g) * 6.28
    cs, sn = ang.cos().cuda(), ang.sin().cuda()
    decay = torch.tensor([0.6, 0.99, 0.9995])
    res = []
    for chunk in (False, True):
        c = StateCache([CacheSpec(slots={"state": ((H, N, P), torch.float32)})], 32, 2, torch.bfloat16, "cuda")
        c.add_sequence(0)
        c.slots[0]["state"].normal_(generator=torch.Generator(device="cuda").manual_seed(1))
        c.slots[0]["state"] *= 30
        c.prepare([0], [9])                                  # the state counts: the portion starts at position 9
        group, _ = split_groups(c.prepare([0], [T]), 1 << 30)
        y = torch.zeros(T, H * P, dtype=torch.bfloat16, device="cuda")
        fn, d = (nat.linear_chunk, decay.double().log2().float()) if chunk else (nat.linear_scan, decay)
        fn(u, cs, sn, d.cuda(), N ** -0.5, c.slots[0]["state"], group, (H, N, P, N, "half", False), y)
        res.append((y.float(), c.slots[0]["state"][c.slot_of[0]].clone()))
    (ya, sa), (yb, sb) = res
    assert float((ya - yb).norm() / ya.norm()) < 2.5e-3      # bf16 outputs
    for h in range(H):
        assert float((sa[h] - sb[h]).norm() / sa[h].norm()) < 2e-5


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [
    attn(6, 2, 20, 40, 12), attn(3, 1, 11, 9, 6), attn(1, 1, 8, 1, 2), attn(4, 4, 64, 64, 64, base=1e6), attn(8, 2, 96, 65, 32),
    attn(10, 1, 128, 128, 96), attn(2, 1, 192, 63, 192), attn(4, 2, 256, 100, 128), attn(2, 1, 264, 70, 2), attn(24, 1, 32, 2, 16),
    attn(2, 2, 30, 1000, 0), attn(2, 1, 600, 90, 64)], ids=_id)
def test_window_attention_mixer(dtype, m):
    mix, p, model = _mixer(m, 48, dtype, 1)
    h = torch.randn(200, 48, generator=torch.Generator().manual_seed(4)).to(dtype)
    run = lambda: O.window_attention(h.double(), p, "l0.mix.", m, 1e-5)      # noqa: E731
    want = run()
    tol = bf16_bound(run, want) if dtype == torch.bfloat16 else FP32
    for sizes in PORTIONS:
        assert err(_run_mixer(mix, model, h.cuda(), sizes), want) < tol, sizes


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [64, 65, 100, 127, 128, 129, 300])
def test_window_edges(dtype, window):
    """Every query asks for one key that stands out: the token itself, the last one of the window, the first one outside, both
    sides of page borders, the first tokens. What is seen is that key's value; what is not seen is not."""
    D, T = 64, 420
    m = attn(2, 1, D, window, 0, scale=1.0)
    mix, _, model = _mixer(m, 2 * D, dtype, 0)
    eye = torch.eye(2 * D).to(dtype)
    with torch.no_grad():                                    # both heads ask with the first half, keys and values are the second
        mix.w_in[:D], mix.w_in[D:2 * D], mix.w_in[2 * D:3 * D] = eye[:D], eye[:D], eye[D:]
        mix.w_o.zero_()
        mix.w_o[:D, :D] = torch.eye(D).to(dtype)
    keys = torch.randn(T, D, generator=torch.Generator().manual_seed(1)).sign()      # unit rms, dot products far below D
    back = [0, 1, window - 1, window, 63, 64, window - 2, window + 1, 65, window // 2]
    dist = torch.tensor([back[i % len(back)] if back[i % len(back)] <= i else (i if i % 2 else 0) for i in range(T)])
    ask = keys[torch.arange(T) - dist]
    h = torch.cat([ask, keys], 1).to(dtype).cuda()
    for sizes in ([T], [T - 40, 1], [30, 2, 17, 64, 1, 90, 3], [1]):
        got = _run_mixer(mix, model, h, sizes)[:, :D].float().cpu()
        like = (got * ask).mean(1)
        assert float(like[dist < window].min()) > 0.9, sizes
        assert float(like[dist >= window].max()) < 0.9 if bool((dist >= window).any()) else window > 255, sizes


@gpu
def test_far_tokens_reach_through_the_state():
    """A slow decay keeps a key that stands out: hundreds of tokens and many portions later its value is what comes out."""
    N, P, T = 32, 32, 700
    m = retention(N, P, [0.9999], 0)
    mix, _, model = _mixer(m, 3 * N + 8, torch.float32, 0)
    W = 3 * N + 8
    with torch.no_grad():
        mix.w_in.zero_()
        for part in range(3):                                # q, k, v: three pieces of the token vector
            mix.w_in[part * N:(part + 1) * N, part * N:(part + 1) * N] = torch.eye(N)
        mix.w_in[3 * N:4 * N, 3 * N] = 1.0                   # a gate of silu(1)
        mix.w_o[:P] = torch.eye(P)
    g = torch.Generator().manual_seed(3)
    k, v = torch.zeros(T, N), torch.randn(T, P, generator=g)
    k[[0, 1, 63, 64, 130], [0, 1, 2, 3, 4]] = 50.0           # five tokens write to rows of their own, the others nothing
    q = torch.zeros(T, N)
    q[torch.arange(T), torch.arange(T) % 5] = 1.0
    h = torch.cat([q, k, v, torch.ones(T, 8)], 1)
    src = torch.tensor([0, 1, 63, 64, 130])[torch.arange(T) % 5]
    want = O.unit_rms(v[src], 1e-5) * (1 / (1 + torch.exp(torch.tensor(-1.0))))
    for sizes in ([T], [64], [300, 1, 2, 100]):
        got = _run_mixer(mix, model, h.cuda(), sizes)[:, :P].cpu()
        assert torch.allclose(got[140:], want[140:], atol=2e-3), sizes
    assert W == h.shape[1]


# ------------------------------------------------------------------------------------------- whole models
@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(MODELS))
def test_model_whole_portions_and_decoding(name, dtype):
    cfg, m = built(name, dtype)
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
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_stream_after_every_layer_run(name):
    cfg, m = built(name)
    toks = tokens(70, cfg["vocab"], 8)
    want = O.forward(toks, weights64(name), cfg)[1]
    c = m.new_cache(2, max_seqs=1)
    c.add_sequence(0)
    seen = []
    m.forward_paged(torch.tensor(toks, device="cuda"), c, c.prepare([0], [70]), on_layer=lambda i, x: seen.append(x.clone()))
    assert len(seen) == len(want)
    for a, b in zip(seen, want):
        assert float((a.double().cpu() - b).norm() / b.norm()) < 1e-5


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name,blocks", [("mixed", 8), ("pages", 8)])
def test_mixed_batches_with_recycled_pages_and_slots(name, blocks, dtype):
    """Four live requests of unequal lengths, portions beside single tokens, pauses, ends and new requests in used pages and
    slots (overwritten with large values in between); every logit equals the request's own."""
    cfg, m = built(name, dtype)
    lens = {"a": 150, "b": 40, "c": 97, "d": 130, "e": 64, "f": 21, "g": 3}
    req = {k: tokens(n, cfg["vocab"], 10 + i) for i, (k, n) in enumerate(lens.items())}
    plan = [  # one dict per step: request -> number of tokens
        {"a": 2, "b": 30, "c": 1}, {"a": 70, "b": 1, "d": 64}, {"a": 1, "c": 60, "d": 1}, {"b": 1, "d": 1}, {"a": 20, "b": 8, "c": 2, "d": 1},
        {"a": 1, "c": 1, "d": 1, "e": 63}, {"a": 40, "d": 5, "e": 1}, {"a": 15, "c": 33, "d": 57, "f": 18}, {"a": 1, "f": 1}, {"f": 2, "g": 2},
        {"g": 1}]
    gen = generator(m, blocks=blocks, max_seqs=4)
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
                c, pages, slot = gen.cache, [b for b in gen.cache.seqs[seq[k]].blocks if b >= 0], gen.cache.slot_of[seq[k]]
                c.free_sequence(seq[k])
                for t in c.pages.values():
                    t[pages] = 50.0
                for d in c.slots.values():
                    for t in d.values():
                        t[slot] = 50.0
    assert all(at[k] == len(req[k]) for k in req) and gen.cache.num_free() == blocks and gen.cache.can_admit()
    for k in req:
        assert err(torch.cat(got[k]), oracle(name, req[k])) < bound(name, req[k], dtype), k


@gpu
@pytest.mark.parametrize("graphs", [True, False])
def test_long_decoding_in_a_batch(graphs):
    """Three requests decode 170 tokens together (fp32, captured steps or eager), crossing page borders and leaving their windows
    behind at different steps."""
    cfg, m = built("mixed")
    gen = generator(m, blocks=12, max_seqs=3, cuda_graphs=graphs)
    req = [tokens(n, cfg["vocab"], 20 + n) for n in (180, 233, 171)]
    seqs = [gen.new_seq() for _ in req]
    gen.prefill(seqs, [r[:len(r) - 170] for r in req])
    got = [gen.step(seqs, [[r[len(r) - 170 + i]] for r in req]).cpu() for i in range(170)]
    assert (gen._graphed is not None) == graphs and gen.cache.seqs[seqs[1]].blocks[0] == -1
    for j, r in enumerate(req):
        assert err(torch.stack([g[j] for g in got]), oracle("mixed", r)[-170:]) < FP32


def _greedy(name, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(O.forward(seq, weights64(name), MODELS[name])[0][-1].argmax()))
    return seq[len(prompt):]


@gpu
def test_greedy_generation_through_the_engine():
    """More requests than slots; prompts longer than a prefill portion run beside decoding slots in one batch."""
    from pmetal_b200.models.generation import Generator
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    cfg, m = built("ones")
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
    g = Generator(m, cache=m.new_cache(16, max_seqs=6))
    res = g.generate(prompts[:2], SamplingParams.greedy(8), num_return_sequences=3)      # forks share pages, copy states
    assert res.tokens == [want[0]] * 3 + [want[1]] * 3
    assert list(g.stream(prompts[3], SamplingParams.greedy(8))) == want[3]
    assert len(g.cache.free_slots) == 6 and g.cache.num_free() == 16


@gpu
def test_sampled_requests_and_background_thread():
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine
    _, m = built("odd", torch.bfloat16)
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
    m = build_model(copy.deepcopy(PRESETS["resevik-tiny"]), torch.float32, "cpu").init_weights(0.05, 3)
    save_pretrained(m, str(tmp_path))
    assert main(["infer", "-m", str(tmp_path), "-p", "hello", "--greedy", "--max-tokens", "5", "--json", "--kv-blocks", "16"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["generated_tokens"] == 5 and out["prompt_tokens"] == 5
    assert main(["infer", "-m", "random:resevik-tiny", "-p", "hi", "--profile-layers", "--json"]) == 0
    assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["layers"]) == 7      # one entry per layer run
    data = tmp_path / "d.jsonl"
    data.write_text('{"text": "some words"}\n{"text": "and a few more"}\n')
    assert main(["eval", "-m", str(tmp_path), "-d", str(data)]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["perplexity"] > 1
    with pytest.raises(SystemExit, match="--lora"):
        main(["infer", "-m", str(tmp_path), "-p", "x", "-l", str(tmp_path)])


@gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(tmp_path, monkeypatch, capsys, dtype):
    """Steps on standard input, logits in files; the pool holds just what the live requests need."""
    import numpy as np
    from pmetal_b200.serve import trace
    cfg = MODELS["mixed"]
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
