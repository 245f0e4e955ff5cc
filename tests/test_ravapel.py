"""Ravapel on the hybrid decoder: kernels and mixers against the plain statement in ``ravapel_oracle.py``, then whole models through
the generator's step function, the state cache, the batching engine and the command line."""
import copy
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import ravapel_oracle as O
from test_hybrid_decoder import FP32, PORTIONS, feed, generator, tokens

from pmetal_b200.models.architectures import build_model, family_of
from pmetal_b200.models.hybrid_decoder import PRESETS, HybridArgs, HybridDecoderLM
from pmetal_b200.models.kv_cache import BLOCK
from pmetal_b200.models.loader import load_pretrained, save_pretrained
from pmetal_b200.models.state_cache import StateCache

gpu = pytest.mark.gpu


# ------------------------------------------------------------------------------------------- models of the tests
def gates(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def chunked(heads, kv, dim, vdim, size, rot, base=10000.0, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": {"base": base, "dims": rot},
            "scale": scale or 1.5 * dim ** -0.5}


def memory(heads, dim, vdim, cap=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def both(left, right, a=0.9, b=1.3):
    return {"left": left, "right": right, "left_scale": a, "right_scale": b}


def kind(m):
    return "parallel" if "left" in m else "hgrn2"


def config(layers, width=48, vocab=101, eps=1e-5, taps=3, loop=None, pair=(131, 17, 3), positions=420):
    """layers: (mixer, width of the feed-forward or None)."""
    d = {"architecture": "Ravapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
         "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pair))}, "max_positions": positions,
         "layers": [{"type": kind(m), "mixer": m, "mlp": f and {"kind": "dense", "ff": f}} for m, f in layers]}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


MODELS = {
    # both mixers, different chunks, one layer without feed-forward, a looped span in the middle
    "mixed": config([(both(chunked(4, 2, 24, 40, 40, 16), memory(3, 16, 24)), 72), (gates(3, 24, 20), 56), (gates(2, 16, 32), None),
                     (both(chunked(3, 3, 20, 16, 70, 8, base=500.0), memory(2, 40, 12, cap=3.0), 1.4, 0.6), 40)], loop=(1, 3, 2)),
    # sizes that are not multiples of what the fast kernels copy at a time; the whole stack runs three times
    "odd": config([(both(chunked(5, 1, 11, 7, 23, 6, base=37.0), memory(3, 7, 5, cap=2.0)), 33), (gates(3, 9, 11), 21)], width=42, vocab=77,
                  eps=1e-3, taps=5, loop=(0, 2, 3), pair=(7, 2, 11)),
    # everything that may be one or nothing, no loop (a large eps: the norm of a single channel is its sign otherwise)
    "ones": config([(gates(1, 1, 1), 1), (both(chunked(1, 1, 2, 1, 1, 2), memory(1, 1, 1), 1.0, 1.0), None),
                    (both(chunked(2, 2, 1, 8, 64, 0), memory(1, 8, 1), -1.0, 1.0), 8)], width=32, vocab=40, eps=0.1, taps=1, pair=(1, 1, 1)),
    # a pass of one layer, heads and states wider than the instances of the tensor-core kernels
    "wide": config([(gates(2, 136, 72), 64), (both(chunked(4, 2, 136, 72, 100, 40), memory(1, 200, 40)), 24), (gates(1, 264, 40), None),
                    (both(chunked(6, 1, 40, 264, 128, 40), memory(2, 264, 136)), 32), (gates(5, 64, 8), 16)], width=64, vocab=90, taps=2,
                   loop=(2, 3, 1)),
}


def random_weights(cfg, seed=0):
    """bf16-representable weights; gates on both sides of one half, some of them nearly shut or nearly open, some bounds zero."""
    g = torch.Generator().manual_seed(seed)
    sd = {}
    for name, shape, _, _ in HybridDecoderLM(HybridArgs.from_dict(cfg), device="meta").named_weights():
        leaf, parts = name.rsplit(".", 1)[-1], name.split(".")
        n = lambda s=1.0: torch.randn(shape, generator=g) * s      # noqa: E731
        u = lambda a, b: torch.rand(shape, generator=g) * (b - a) + a      # noqa: E731
        if leaf in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            t = u(-0.5, 0.5)
        elif leaf == "norm":
            t = u(0.6, 1.4)
        elif leaf == "lower":
            t = u(-0.3, 0.9).clamp_min(0)
        elif leaf == "pb":
            t = u(-4.0, -1.0)
        elif leaf == "canon1":
            t = n(0.35)
        elif leaf == "b":
            t = {"f": u(0.0, 6.0) if "right" in parts else n(2.5), "i": n()}.get(parts[-2], n(0.2))
        elif leaf in ("embed", "bigram", "pos"):
            t = n({"embed": 1.0, "bigram": 0.6, "pos": 0.4}[leaf])
        else:
            t = n(shape[1] ** -0.5)
        sd[name] = t.to(torch.bfloat16)
    return sd


_CACHE = {}


def cached(key, make):
    if key not in _CACHE:
        _CACHE[key] = make()
    return _CACHE[key]


def weights16(name):
    return cached(("w16", name), lambda: random_weights(MODELS[name]))


def weights64(name):
    return cached(("w", name), lambda: {k: v.double() for k, v in weights16(name).items()})


def built(name, dtype=torch.float32, device="cuda"):
    def make():
        m = build_model(MODELS[name], dtype, device)
        assert m.load_hf_state_dict(weights16(name)) == []
        return m.eval()
    return MODELS[name], cached(("m", name, dtype, device), make)


def oracle(name, toks):
    return cached(("o", name, tuple(toks)), lambda: O.forward(toks, weights64(name), MODELS[name])[0])


def row_errors(got, want):
    """Root mean square of every row's difference (mean taken off) over that of the expected rows."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


def row_limits(run, want, dtype):
    """What each row may differ by. bf16: three times what rounding the oracle's own projections and activations does to that row (the
    largest of several roundings; some rows are divided by what nearly cancels), at least what it does to the middle row, plus a
    little. fp32: ``run(torch.float32)`` in place of the roundings, no row below the usual tolerance."""
    if dtype == torch.float32:
        return (6 * row_errors(run(torch.float32), want)).clamp_min(FP32)
    e = []
    for seed in (None, 1, 2, 3):
        with O.rounding(seed):
            e.append(row_errors(run(torch.float64), want))
    e = torch.stack(e).amax(0)
    return 3 * torch.maximum(e, e.median()) + 2e-3


def worst(got, want, limits):
    return float((row_errors(got, want) / limits).max())


def limits(name, toks, dtype):
    w = lambda t: {k: v.to(t) for k, v in weights16(name).items()}      # noqa: E731
    return cached(("b", name, tuple(toks), dtype),
                  lambda: row_limits(lambda t: O.forward(toks, w(t), MODELS[name])[0], oracle(name, toks), dtype))


# ------------------------------------------------------------------------------------------- host side (no GPU)
def test_registry_and_configuration():
    cfg = MODELS["mixed"]
    assert family_of(cfg) == "hybrid" and family_of({"model_type": "ravapel"}) == "hybrid"
    a = HybridArgs.from_dict(cfg)
    assert (a.vocab_size, a.hidden_size, a.num_hidden_layers, a.norm_eps, a.taps, a.max_positions) == (101, 48, 4, 1e-5, 3, 420)
    assert a.pair == (131, 17, 3) and a.loop == (1, 3, 2) and a.to_hf_dict() == cfg
    assert a.runs == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]      # the first pass is entered like the others
    assert HybridArgs.from_dict(MODELS["ones"]).runs == [(0, False), (1, False), (2, False)]
    assert HybridArgs.from_dict(dict(MODELS["ones"], loop=None)).loop is None
    m = build_model(cfg, torch.float32, "cpu")
    assert isinstance(m, HybridDecoderLM) and m.norm_b is None and m.head is not m.embed_tokens
    shapes = {n: tuple(s) for n, s, *_ in m.named_weights()}
    assert shapes["bigram"] == (132, 48) and shapes["pos"] == (420, 48) and shapes["loop.in"] == (48, 96) and shapes["l3.canon1"] == (48, 3)
    assert shapes["l0.mix.left.q"] == (96, 48) and shapes["l0.mix.left.pb"] == (4,) and shapes["l0.mix.left.k.norm"] == (24,)
    assert shapes["l0.mix.right.i"] == (3, 48) and shapes["l0.mix.right.f.b"] == (3,) and shapes["l0.mix.right.norm"] == (72,)
    assert shapes["l1.mix.lower"] == (72,) and shapes["l1.mix.norm"] == (20,) and shapes["l1.mlp.up.b"] == (56,)
    assert "l2.norm2" not in shapes and "l2.norm2b" not in shapes and "l2.norm1b" in shapes and not any(n.startswith("l2.mlp") for n in shapes)
    assert "loop.in" not in {n for n, *_ in build_model(MODELS["ones"], torch.float32, "cpu").named_weights()}
    c = m.new_cache(4, max_seqs=2)
    assert sorted(c.pages) == [0, 5] and sorted(c.slots) == [0, 1, 2, 3, 4, 5, 6] and c.window == 70 and not c.can_truncate
    assert c.pages[0].shape == (5, BLOCK, 2 * (24 + 40)) and set(c.slots[0]) == {"state", "norm", "max", "canon"} and set(c.slots[6]) == {"token"}
    assert c.slots[0]["max"].shape == (3, 3, 6) and c.slots[1]["state"].shape == (3, 3, 24, 20) and c.slots[4]["canon"].shape == (3, 2, 48)
    assert all(t.dtype == torch.float32 for k in (0, 1) for n, t in build_model(cfg, torch.bfloat16, "cpu").new_cache(4).slots[k].items() if n != "canon")
    with pytest.raises(RuntimeError, match="CUDA"):
        m(torch.tensor([1, 2]))


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "key/value"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("mask"), "mask"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(mask=None), "mask"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(mask={"size": 0}), "mask"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26), "rot"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=3.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"].update(heads=0), "positive"),
    (lambda c: c["layers"][1]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][1].update(type="lightning"), "unknown mixer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "feed-forward"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["canon"].update(taps=0), "taps"),
    (lambda c: c["canon"].update(taps=18), "taps"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "pair"),
    (lambda c: c.update(max_positions=0), "max_positions"),
])
def test_bad_configurations_are_refused(change, what):
    c = copy.deepcopy(MODELS["mixed"])
    change(c)
    with pytest.raises(ValueError, match=what):
        HybridArgs.from_dict(c)


def test_checkpoint_round_trip(tmp_path):
    cfg, sd = MODELS["odd"], weights16("odd")
    m = build_model(cfg, torch.bfloat16, "cpu")
    m.load_hf_state_dict(sd)
    save_pretrained(m, str(tmp_path))
    for dtype in (torch.bfloat16, torch.float32):
        back, args, mdir = load_pretrained(str(tmp_path), dtype)
        assert mdir == str(tmp_path) and args.to_hf_dict() == cfg
        got = back.hf_state_dict()
        assert set(got) == set(sd) and all(torch.equal(got[k], sd[k]) for k in sd)
    with pytest.raises(KeyError, match="l0.mix.right.i.b"):
        m.load_hf_state_dict({k: v for k, v in sd.items() if k != "l0.mix.right.i.b"})
    with pytest.raises(ValueError, match="shape"):
        m.load_hf_state_dict(dict(sd, **{"l1.canon1": torch.zeros(5, 42)}))


def test_sequences_end_with_the_position_table():
    c = build_model(MODELS["ones"], torch.float32, "cpu").new_cache(16, max_seqs=2)
    assert c.max_length == 420
    c.add_sequence(0)
    c.reserve(0, 420)
    with pytest.raises(ValueError, match="420 positions"):
        c.reserve(0, 1)
    assert c.length(0) == 420 and StateCache([], 4, 2, torch.float32, "cpu").max_length == 0


def test_engine_and_presets_build():
    from pmetal_b200 import build
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    m = build_model(MODELS["ones"], torch.float32, "cpu")
    e = ContinuousBatchEngine(m, max_slots=3, num_blocks=64)
    assert e.mixed and e.prefix is None
    late = e.submit(Request([1] * 421, SamplingParams.greedy(1)))
    for _ in range(5):
        e.submit(Request([1, 2, 3]))
    e._admit()
    assert len(e.slots) == 3 and late.finish_reason == "error:too_long"      # more tokens than positions
    for p in ("ravapel-tiny", "ravapel-1b", "ravapel-2b"):
        HybridDecoderLM(HybridArgs.from_dict(PRESETS[p]), torch.bfloat16, "meta")
    a, args, d = load_pretrained("random:ravapel-tiny", torch.float32)
    assert d is None and args.model_type == "ravapel" and float(a.embed_tokens.abs().sum()) > 0
    assert float(a.norm_w.abs().sum()) == 0 and float(a.layers[0].mixer.norm_w.min()) == 1      # norms around zero and around one
    assert float(a.layers[1].mixer.right.g_bias[3:].min()) >= 1 and float(a.layers[1].mixer.right.g_bias[:3].abs().max()) == 0
    assert all(os.path.exists(os.path.join(build.CSRC, s + ".cu")) for s in build.COMPONENTS["ravapel"])


def _mix(change):
    """cfg with ``change`` applied to a copy of every mixer entry of the parallel layers."""
    def run(cfg):
        c = copy.deepcopy(cfg)
        for l in c["layers"]:
            if l["type"] == "parallel":
                change(l["mixer"])
        return c
    return run


def _weights(change):
    """Weights in which ``change(name, tensor)`` replaces some."""
    def run(p):
        return {k: v if (t := change(k, v)) is None else t for k, v in p.items()}
    return run


def _planted(monkeypatch, what, cfg, p):
    """Makes one mistake in the oracle; returns the configuration and weights to run it with."""
    real = {n: getattr(O, n) for n in ("embedding", "input_convolution", "forget", "gated_state", "rotate_halves", "visible", "sigmoid_attend",
                                       "matrix_memory", "memory_gates", "centred_norm", "unit_rms", "enter_pass", "layer", "gated_mlp")}
    put = lambda n, f: monkeypatch.setattr(O, n, f)      # noqa: E731
    if what in ("scales swapped", "no score factor", "rotation of all channels", "base of another layer"):
        change = {"scales swapped": lambda m: m.update(left_scale=m["right_scale"], right_scale=m["left_scale"]),
                  "no score factor": lambda m: m["left"].update(scale=1.0),
                  "rotation of all channels": lambda m: m["left"]["rot"].update(dims=m["left"]["dim"]),
                  "base of another layer": lambda m: m["left"]["rot"].update(base=10000.0 + 500.0 - m["left"]["rot"]["base"])}[what]
        return _mix(change)(cfg), p
    if what == "one pass":
        return dict(cfg, loop=dict(cfg["loop"], times=1)), p
    if what == "factors of the pair swapped":
        e = cfg["embedding"]["bigram"]
        return dict(cfg, embedding={"bigram": dict(e, mul_prev=e["mul_cur"], mul_cur=e["mul_prev"])}), p
    zero = {"no position rows": ("pos",), "no pair rows": ("bigram",), "no score bias": (".pb",), "no bound": (".lower",), "no gate bias": ("mix.f.b",),
            "no bias of the input gate": (".i.b",), "no bias of the forget gate": ("right.f.b",), "no feed-forward biases": ("gate.b", "up.b", "down.b"),
            "no convolution": ("canon1",)}.get(what)
    if zero:
        return cfg, _weights(lambda n, t: torch.zeros_like(t) if n.endswith(zero) and not (what == "no gate bias" and "right" in n) else None)(p)
    if what == "first token paired with token 0":
        put("embedding", lambda toks, p, cfg: torch.cat([real["embedding"]([0] + list(toks), dict(p, pos=p["pos"].roll(1, 0)), cfg)[1:]]))
    elif what == "positions one late":
        return cfg, dict(p, pos=p["pos"].roll(1, 0))
    elif what == "convolution reversed":
        put("input_convolution", lambda h, w: real["input_convolution"](h, w.flip(1)))
    elif what == "convolution one token late":
        put("input_convolution", lambda h, w: h + torch.cat([h[:1] * 0, (real["input_convolution"](h, w) - h)[:-1]]))
    elif what == "convolution in place of the input":
        put("input_convolution", lambda h, w: real["input_convolution"](h, w) - h)
    elif what == "write by one":
        put("gated_state", lambda q, f, v: real["gated_state"](q, f, v / (1 - f).mean(-1, keepdim=True)))
    elif what == "gate behind the write":
        put("gated_state", lambda q, f, v: real["gated_state"](q * f, f, v))
    elif what == "state lost at token 64":
        put("gated_state", lambda q, f, v: torch.cat([real["gated_state"](q[:64], f[:64], v[:64]), real["gated_state"](q[64:], f[64:], v[64:])]))
    elif what == "window in place of the chunk":
        def seen(T, chunk):
            d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
            return (d >= 0) & (d < chunk)
        put("visible", seen)
    elif what == "chunks one token late":
        put("visible", lambda T, chunk: real["visible"](T + 1, chunk)[1:, 1:])
    elif what == "weights divided by their sum":
        def attend(q, k, v, scale, bias, seen):
            w = torch.sigmoid((q @ k.t()) * scale + bias) * seen
            return w @ v / w.sum(-1, keepdim=True)
        put("sigmoid_attend", attend)
    elif what == "key of the wrong group":
        put("sigmoid_attend", lambda q, k, v, scale, bias, seen: real["sigmoid_attend"](q, k.roll(1, -1), v, scale, bias, seen))
    elif what == "pairs rotated":
        def rot(x, base, dims):
            ix = [i // 2 + (i % 2) * (dims // 2) for i in range(dims)]
            y = x.clone()
            y[:, :, ix] = x[:, :, :dims]
            y = real["rotate_halves"](y, base, dims)
            out = y.clone()
            out[:, :, :dims] = y[:, :, ix]
            return out
        put("rotate_halves", rot)
    elif what == "maximum from minus infinity":
        def mem(q, k, v, i, f):
            N, P = q.shape[1], v.shape[1]
            S, n, m, out = torch.zeros(N, P, dtype=q.dtype), torch.zeros(N, dtype=q.dtype), torch.tensor(-1e9, dtype=q.dtype), []
            for t in range(q.shape[0]):
                new = torch.maximum(f[t] + m, i[t])
                S = torch.exp(f[t] + m - new) * S + torch.exp(i[t] - new) * k[t][:, None] * v[t]
                n = torch.exp(f[t] + m - new) * n + torch.exp(i[t] - new) * k[t]
                m = new
                out.append((q[t] @ S) / (torch.maximum((n @ q[t]).abs(), torch.ones(())) + 1e-6))
            return torch.stack(out)
        put("matrix_memory", mem)
    elif what == "normaliser without bound":
        def mem(q, k, v, i, f):
            one = real["matrix_memory"](q, k, torch.ones_like(v[:, :1]), i, f)      # n . q over the divisor
            return real["matrix_memory"](q, k, v, i, f) / one.abs().clamp_min(1e-3)
        put("matrix_memory", mem)
    elif what == "no cap":
        put("memory_gates", lambda h, p, pre, cap: real["memory_gates"](h, p, pre, 1e4))
    elif what == "sigmoid of the forget gate":
        put("memory_gates", lambda h, p, pre, cap: (real["memory_gates"](h, p, pre, cap)[0], -torch.exp(real["memory_gates"](h, p, pre, cap)[1])))
    elif what == "norm weight without one":
        put("centred_norm", lambda x, w, eps: real["unit_rms"](x, eps) * (0.3 + w))
    elif what == "no norm behind the mixer":
        def layer(x, i, spec, p, eps):
            pre = f"l{i}."
            h = O.input_convolution(O.centred_norm(x, p[pre + "norm1"], eps), p[pre + "canon1"])
            x = x + (O.hgrn2 if spec["type"] == "hgrn2" else O.parallel)(h, p, pre + "mix.", spec["mixer"], eps)
            if spec.get("mlp") is not None:
                x = x + O.centred_norm(O.gated_mlp(O.centred_norm(x, p[pre + "norm2"], eps), p, pre + "mlp."), p[pre + "norm2b"], eps)
            return x
        put("layer", layer)
    elif what == "embedding output in front":
        put("enter_pass", lambda x, x0, w: real["enter_pass"](x0, x, w))
    elif what == "first pass not entered":
        count = []
        def enter(x, x0, w):
            count.append(1)
            return x if len(count) == 1 else real["enter_pass"](x, x0, w)
        put("enter_pass", enter)
    elif what == "activation on the other half":
        put("gated_mlp", lambda h, p, pre: real["gated_mlp"](h, {k.replace("gate", "#").replace("up", "gate").replace("#", "up"): v
                                                                  for k, v in p.items() if k.startswith(pre)}, pre))
    return cfg, p


FAULTS = ["scales swapped", "no score factor", "rotation of all channels", "base of another layer", "one pass", "factors of the pair swapped",
          "no position rows", "no pair rows", "no score bias", "no bound", "no gate bias", "no bias of the input gate",
          "no bias of the forget gate", "no feed-forward biases", "no convolution", "first token paired with token 0", "positions one late",
          "convolution reversed", "convolution one token late", "convolution in place of the input", "write by one", "gate behind the write",
          "state lost at token 64", "window in place of the chunk", "chunks one token late", "weights divided by their sum",
          "key of the wrong group", "pairs rotated", "maximum from minus infinity", "normaliser without bound", "no cap",
          "sigmoid of the forget gate", "norm weight without one", "no norm behind the mixer", "embedding output in front",
          "first pass not entered", "activation on the other half"]


@pytest.mark.parametrize("what", FAULTS)
def test_faults_show_in_the_test_model(monkeypatch, what):
    """The model the comparisons below use makes each of these mistakes visible, well above the bf16 tolerance."""
    toks = tokens(150, 101, 5)
    want, tol = oracle("mixed", toks), limits("mixed", toks, torch.bfloat16)
    cfg, p = _planted(monkeypatch, what, MODELS["mixed"], weights64("mixed"))
    assert worst(O.forward(toks, p, cfg)[0], want, tol) > 1.5


# ------------------------------------------------------------------------------------------- kernels
def _meta(cache, seqs, counts):
    for s in seqs:
        if s not in cache.seqs:
            cache.add_sequence(s)
    return cache.prepare(seqs, counts)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,taps", [(48, 3), (42, 5), (1000, 4), (2560, 2), (24, 1), (40, 17)])
def test_input_convolution(dtype, width, taps):
    """Three sequences in portions of unequal sizes, in used rings; the single-token form of the norm kernel beside the kernel for
    longer portions."""
    from pmetal_b200.models.state_cache import CacheSpec
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(width)
    lens = (90, 41, 26)
    hs = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    w = torch.randn(width, taps, generator=g) * 0.4
    want = [O.input_convolution(h.double(), w.double()) for h in hs]
    c = StateCache([CacheSpec(slots={"canon": ((taps - 1, width), None)})], 16, 4, dtype, "cuda")
    ring = c.slots[0]["canon"]
    ring.fill_(9.0)
    c.add_sequence(7)                                        # the others do not sit in the first slots
    wt, at, got = w.t().contiguous().cuda(), [0, 0, 0], [[], [], []]
    zero = torch.zeros(width, device="cuda")
    for sizes in ((1, 0, 2), (1, 1, 0), (40, 1, 1), (1, 1, 1), (0, 2, 16), (20, 33, 1), (2, 1, 4), (1, 1, 0), (0, 0, 1), (24, 1, 0)):
        seqs = [i for i in range(3) if sizes[i]]
        meta = _meta(c, seqs, [sizes[i] for i in seqs])
        h = torch.cat([hs[i][at[i]:at[i] + sizes[i]] for i in seqs]).cuda()
        if meta.max_q == 1:                                  # rows whose root mean square is one pass the norm unchanged, up to rounding
            x = h.float()
            scale = x.pow(2).mean(1, keepdim=True).sqrt()
            conv = (wt, ring, meta.state_slots, meta.positions)
            _, out = nat.branch_norm(x / scale, 0.0, 1.0, wn=zero, dtype=dtype, conv=conv)
            want_ring = (x / scale).to(dtype)
            for j, i in enumerate(seqs):                     # the ring and the oracle take the normed row
                hs[i][at[i]] = want_ring[j].cpu()
                want[i] = O.input_convolution(hs[i].double(), w.double())
        else:
            out = nat.canon(h, wt, ring, meta)
        o = 0
        for i in seqs:
            got[i].append(out[o:o + sizes[i]].cpu().double())
            at[i] += sizes[i]
            o += sizes[i]
    assert tuple(at) == lens
    for i in range(3):
        torch.testing.assert_close(torch.cat(got[i]), want[i], **(dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=1e-5, atol=1e-5)))


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 42, 999, 2560, 8192])
def test_norms_on_both_sides_of_a_sum(dtype, width):
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)
    for n in (3, 400):
        x, wb, wn, bias, ybuf = r(n, width) * 3, r(width) * 0.3, r(width) * 0.3, r(width), r(n, width + 8).to(dtype)
        y = ybuf.cuda()[:, :width]
        s = ybuf[:, :width].double() + bias.double()
        v = x.double() + O.centred_norm(s, wb.double(), 1e-3)
        xs = x.cuda()
        of, oc = nat.branch_norm(xs, 1e-3, 1.0, y=y, bias=bias.cuda(), wb=wb.cuda(), wn=wn.cuda(), out=xs)
        assert of is xs and oc.dtype == dtype
        torch.testing.assert_close(of.cpu().double(), v, rtol=2e-5, atol=2e-5)
        torch.testing.assert_close(oc.cpu().double(), O.centred_norm(v, wn.double(), 1e-3), **tol)
        cat = torch.full((n, 2 * width), 7.0, dtype=dtype, device="cuda")      # the sum itself, beside other columns
        of, oc = nat.branch_norm(x.cuda(), 1e-3, 1.0, y=y, bias=bias.cuda(), wb=wb.cuda(), oc=cat[:, :width])
        torch.testing.assert_close(cat[:, :width].cpu().double(), v, **tol)
        assert bool((cat[:, width:] == 7).all())
        rows = torch.tensor([n - 1, 0])
        of, oc = nat.branch_norm(x.cuda(), 1e-3, 0.0, y=y, wb=wb.cuda(), wn=wn.cuda(), rows=rows.cuda(), want_stream=False)
        v = x.double() + O.unit_rms(ybuf[:, :width].double(), 1e-3) * wb.double()
        assert of is None and oc.shape == (2, width)
        torch.testing.assert_close(oc.cpu().double(), (O.unit_rms(v, 1e-3) * wn.double())[rows], **tol)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,pair", [(48, (131, 17, 3)), (42, (1, 5, 7)), (64, (100003, 49999, 77777)), (40, (5, 0, 1))])
def test_embedding_of_pairs_and_positions(dtype, width, pair):
    """The previous token comes from the step or from the sequence's slot; products beyond 32 bits."""
    from pmetal_b200.models.state_cache import CacheSpec
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(width)
    vocab, pos = 60001, 200
    p = {"embed": torch.randn(vocab, width, generator=g), "bigram": torch.randn(pair[0] + 1, width, generator=g), "pos": torch.randn(pos, width, generator=g)}
    p = {k: v.to(dtype) for k, v in p.items()}
    cfg = {"embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pair))}}
    c = StateCache([CacheSpec(slots={"token": ((1,), torch.int32)})], 16, 4, dtype, "cuda")
    c.slots[0]["token"].fill_(-5)
    c.add_sequence(9)
    toks = [tokens(n, vocab, n) for n in (90, 30, 5)]
    at, got, cats = [0, 0, 0], [[], [], []], [[], [], []]
    for sizes in ((1, 2, 0), (64, 1, 1), (1, 1, 1), (2, 26, 3), (22, 0, 0)):
        seqs = [i for i in range(3) if sizes[i]]
        meta = _meta(c, seqs, [sizes[i] for i in seqs])
        ids = torch.tensor([t for i in seqs for t in toks[i][at[i]:at[i] + sizes[i]]], device="cuda")
        cat = torch.zeros(ids.shape[0], 2 * width, dtype=dtype, device="cuda")
        out = nat.pair_embed(ids, p["embed"].cuda(), p["bigram"].cuda(), p["pos"].cuda(), meta, c.slots[0]["token"], pair, cat[:, width:])
        o = 0
        for i in seqs:
            got[i].append(out[o:o + sizes[i]].cpu().double())
            cats[i].append(cat[o:o + sizes[i], width:].cpu().double())
            at[i], o = at[i] + sizes[i], o + sizes[i]
        assert bool((cat[:, :width] == 0).all())
    for i, t in enumerate(toks):
        want = O.embedding(t, {k: v.double() for k, v in p.items()}, cfg)
        torch.testing.assert_close(torch.cat(got[i]), want, rtol=1e-6, atol=1e-6)
        torch.testing.assert_close(torch.cat(cats[i]), want, **(dict(rtol=5e-3, atol=1e-3) if dtype == torch.bfloat16 else dict(rtol=1e-6, atol=1e-6)))


@gpu
def test_projection_with_fp32_columns():
    """Activations in bf16, logits of gates in fp32 from one weight: mat-vec with and without tensor cores, GEMM, few and many logits."""
    from pmetal_b200.ops import functional as ops
    g = torch.Generator().manual_seed(0)
    for K in (64, 40, 2048):
        for low, tail in ((64, 6), (200, 72), (8, 200)):
            w = torch.randn(-(-(low + tail) // 8) * 8, K, generator=g).to(torch.bfloat16)
            for T in (1, 4, 11, 16, 17, 300):
                x = torch.randn(T, K, generator=g).to(torch.bfloat16)
                u, z = ops.project_mixed(x.cuda(), w.cuda(), low)
                want = x.double() @ w.double().t()
                assert u.dtype == torch.bfloat16 and z.dtype == torch.float32 and u.shape == (T, low)
                assert float((u.cpu().double() - want[:, :low]).abs().max()) < 5e-3 * K ** 0.5 * 5
                assert float((z.cpu().double()[:, :tail] - want[:, low:low + tail]).abs().max()) < 2e-5 * K ** 0.5


# ------------------------------------------------------------------------------------------- mixers
def _mixer(m, width, dtype, seed, sd=None, **kw):
    cfg = config([(m, None)], width=width, positions=8192, **kw)
    sd = sd or random_weights(cfg, seed)
    model = build_model(cfg, dtype, "cuda")
    model.load_hf_state_dict(sd, strict=False)
    return model.layers[0].mixer, {k: v.double() for k, v in sd.items()}, model


def _run_mixer(mix, model, h, sizes):
    """h [T, width] through the mixer in portions; the sequence sits in shuffled pages and a later slot, which hold what an earlier
    owner may have left."""
    from pmetal_b200.models.mixers import StepContext
    blocks = max(40, h.shape[0] // BLOCK + 2)
    cache = model.new_cache(blocks, max_seqs=3)
    cache.free = [b for b in range(0, blocks, 2)] + [b for b in range(1, blocks, 2)]
    cache.add_sequence(0)
    cache.add_sequence(1)
    for t in list(cache.pages.values()) + [t for n, t in cache.slots[0].items() if n != "canon"]:
        t.fill_(7.0)
    out, at, k = [], 0, 0
    while at < h.shape[0]:
        n = min(sizes[min(k, len(sizes) - 1)], h.shape[0] - at)
        meta = cache.prepare([1], [n])
        out.append(mix(h[at:at + n].contiguous(), cache, StepContext(meta, model._freqs), 0)[:, :h.shape[1]])
        at, k = at + n, k + 1
    return torch.cat(out)


def _id(m):
    if "left" in m:
        a, b = m["left"], m["right"]
        return f"h{a['heads']}g{a['kv_heads']}d{a['dim']}v{a['vdim']}c{a['mask']['size']}-h{b['heads']}d{b['dim']}v{b['vdim']}"
    return f"h{m['heads']}d{m['dim']}v{m['vdim']}"


def _oracle_mixer(m, h, p):
    return (O.hgrn2 if kind(m) == "hgrn2" else O.parallel)(h, p, "l0.mix.", m, 1e-5)


def _compare(m, dtype, h, sd=None, portions=PORTIONS, seed=1):
    mix, p, model = _mixer(m, h.shape[1], dtype, seed, sd)
    run = lambda t: _oracle_mixer(m, h.to(t), {k: v.to(t) for k, v in p.items()})      # noqa: E731
    want = run(torch.float64)
    tol = row_limits(run, want, dtype)
    for sizes in portions:
        assert worst(_run_mixer(mix, model, h.cuda(), sizes), want, tol) < 1, sizes


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [gates(3, 24, 20), gates(3, 9, 11), gates(1, 1, 1), gates(2, 64, 96), gates(4, 32, 33), gates(1, 136, 72), gates(2, 200, 40),
                               gates(1, 256, 64), gates(1, 264, 40), gates(7, 16, 128), gates(1, 128, 300)], ids=_id)
def test_channel_gates(dtype, m):
    _compare(m, dtype, torch.randn(200, 48, generator=torch.Generator().manual_seed(4)).to(dtype))


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shift", [-60.0, -14.0, 12.0])
def test_channel_gates_far_from_one_half(dtype, shift):
    """Gates that shut at once, several in a row (products far below the smallest fp32 number), and gates that stay open for
    thousands of tokens: channels of all kinds beside each other, no bound and a high one."""
    m = gates(2, 40, 24)
    sd = random_weights(config([(m, None)], width=48, positions=8192), 2)
    pick = torch.arange(80) % 3
    sd["l0.mix.f.b"] = torch.where(pick == 0, torch.tensor(shift), torch.where(pick == 1, torch.tensor(3.0), torch.tensor(9.0))).to(torch.bfloat16)
    sd["l0.mix.f"] = (sd["l0.mix.f"].float() * (8 if shift < 0 else 1)).to(torch.bfloat16)
    sd["l0.mix.lower"] = torch.where(torch.arange(80) % 5 == 0, torch.tensor(0.96875), torch.tensor(0.0)).to(torch.bfloat16)
    _compare(m, dtype, torch.randn(700, 48, generator=torch.Generator().manual_seed(3)).to(dtype), sd,
             ([700], [300, 2, 1, 397], [16], [70, 1, 17, 2, 64]))


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [both(chunked(4, 2, 24, 40, 40, 16), memory(3, 16, 24)), both(chunked(5, 1, 11, 7, 23, 6, base=37.0), memory(3, 7, 5, cap=2.0)),
                               both(chunked(1, 1, 2, 1, 1, 2), memory(1, 1, 1), 1.0, 1.0), both(chunked(2, 2, 16, 8, 64, 0), memory(2, 64, 48), -0.7, 0.4),
                               both(chunked(4, 2, 136, 72, 100, 40), memory(1, 200, 40)), both(chunked(6, 1, 40, 264, 1000, 40), memory(1, 264, 136)),
                               both(chunked(8, 8, 64, 64, 128, 64), memory(4, 32, 33, cap=30.0)), both(chunked(2, 1, 600, 8, 50, 600), memory(1, 128, 128)),
                               both(chunked(16, 2, 32, 128, 65, 32, scale=2.0), memory(2, 96, 200))], ids=_id)
def test_attention_beside_a_matrix_memory(dtype, m):
    _compare(m, dtype, torch.randn(200, 48, generator=torch.Generator().manual_seed(5)).to(dtype))


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("what", ["open", "shut", "large"])
def test_memory_gates_at_their_bounds(dtype, what):
    """Input and forget gates at either end of the cap: a memory that keeps nearly everything, one that keeps next to nothing, input
    gates so large that the normaliser's constant counts; more tokens than one pass of the gate kernel takes."""
    m = both(chunked(1, 1, 8, 8, 64, 8), memory(2, 24, 20, cap=14.0), 0.0, 1.0)
    sd = random_weights(config([(m, None)], width=48, positions=8192), 2)
    for gate, b in {"open": (("f", 30.0), ("i", 0.0)), "shut": (("f", -40.0), ("i", -2.0)), "large": (("f", 9.0), ("i", 60.0))}[what]:
        sd[f"l0.mix.right.{gate}.b"] = torch.full((2,), b).to(torch.bfloat16)
    T = 4400 if what == "open" else 600
    _compare(m, dtype, torch.randn(T, 48, generator=torch.Generator().manual_seed(3)).to(dtype), sd,
             ([T], [T - 70, 1, 17, 2, 50]) if what == "open" else ([T], [300, 2, 1, 297], [16], [70, 1, 17, 2, 64]))


def _standout(size, D, T, dtype):
    """(mixer entry, weights, inputs): a token vector is [what it asks for | what it is | its value]; keys are sign vectors and every
    query asks for one key, so that one weight stands far above the others. The memory beside it adds nothing."""
    g = torch.Generator().manual_seed(1)
    W = 3 * D
    eye = lambda at: torch.eye(W)[at * D:(at + 1) * D]      # noqa: E731
    out = torch.zeros(W, D)
    out[:D] = torch.eye(D)
    m = both(chunked(1, 1, D, D, size, 0, scale=0.5), memory(1, 1, 1), 1.0, 0.0)
    p = {"q": eye(0), "k": eye(1), "v": eye(2), "q.norm": torch.ones(D), "k.norm": torch.ones(D), "pb": torch.tensor([-24.0]), "o": out}
    sd = random_weights(config([(m, None)], width=W, positions=8192), 0)
    sd.update({"l0.mix.left." + k: v.to(torch.bfloat16) for k, v in p.items()})
    keys, values = torch.randn(T, D, generator=g).sign(), torch.randn(T, D, generator=g)
    # the token itself, neighbours, page borders, the first key of the chunk, the last one before it, the first token of all
    def asks(i):
        own = i % size
        want = [0, 1, 63, 64, 65, own, own + 1, 127, 128, i][i % 10]
        return min(want, i)
    dist = torch.tensor([asks(i) for i in range(T)])
    h = torch.cat([keys[torch.arange(T) - dist], keys, values], 1).to(dtype)
    return m, sd, h, dist


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("size", [64, 90, 128, 7, 1000])
def test_far_keys_page_borders_and_chunk_edges(dtype, size):
    """Keys just inside a chunk are found, those just outside are not; chunks that do and do not divide into pages."""
    m, sd, h, dist = _standout(size, 64, 420, dtype)
    mix, p, model = _mixer(m, 192, dtype, 0, sd)
    run = lambda x=h: _oracle_mixer(m, x.double(), p)[:, :64]      # noqa: E731
    want = run()
    found = want.norm(dim=1) > 1.0
    inside = dist <= torch.arange(420) % size
    assert torch.equal(found, inside) and bool(inside.any()) and (size == 1000 or bool((~inside).any()))
    scale = float(want[found].norm(dim=1).mean())
    for sizes in ([420], [380, 1], [30, 2, 17, 64, 1, 90, 3], [1], [2], [64], [63, 1, 65]):
        got = _run_mixer(mix, model, h.cuda(), sizes)[:, :64].double().cpu()
        assert float((got - want).norm(dim=1).max()) < (0.03 if dtype == torch.bfloat16 else 1e-4) * scale, sizes


# ------------------------------------------------------------------------------------------- whole models
@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(MODELS))
def test_model_whole_portions_and_decoding(name, dtype):
    cfg, m = built(name, dtype)
    toks = tokens(150, cfg["vocab"], 5)
    want, tol = oracle(name, toks), limits(name, toks, dtype)
    assert worst(m(torch.tensor(toks, device="cuda")), want, tol) < 1
    docs = torch.tensor(toks[:70] + toks, device="cuda")                                  # two documents in one stream
    got = m(docs, cu_seqlens=torch.tensor([0, 70, 220], device="cuda"))
    assert worst(got[:70], want[:70], tol[:70]) < 1 and worst(got[70:], want, tol) < 1
    for sizes in ([150], [130, 1], [2], [1], [64, 1, 1, 63, 3], [5, 20, 70, 2, 1, 1]):
        gen = generator(m)
        got = feed(gen, gen.new_seq(), toks, sizes)
        assert worst(got, want, tol) < 1, sizes
        assert gen.cache.length(0) == 150


@gpu
@pytest.mark.parametrize("name", ["mixed", "odd", "ones"])
def test_stream_after_every_layer_run(name):
    cfg, m = built(name)
    toks = tokens(70, cfg["vocab"], 8)
    want = O.forward(toks, weights64(name), cfg)[1]
    for sizes in ([70], [69, 1]):
        c = m.new_cache(2, max_seqs=1)
        c.add_sequence(0)
        parts, at = [], 0
        for n in sizes:
            seen = []
            m.forward_paged(torch.tensor(toks[at:at + n], device="cuda"), c, c.prepare([0], [n]), on_layer=lambda i, x: seen.append((i, x.clone())))
            assert [i for i, _ in seen] == list(range(len(want)))
            parts.append(torch.stack([x for _, x in seen]))
            at += n
        for a, b in zip(torch.cat(parts, 1), want):
            assert float((a.double().cpu() - b).norm() / b.norm()) < 1e-5


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mixed_batches_with_recycled_pages_and_slots(dtype):
    """Four live requests of unequal lengths, portions beside single tokens, pauses, ends and new requests in used pages and slots
    (overwritten with large values in between); every logit equals the request's own."""
    cfg, m = built("mixed", dtype)
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
                c = gen.cache
                pages, slot = [b for b in c.seqs[seq[k]].blocks if b >= 0], c.slot_of[seq[k]]
                c.free_sequence(seq[k])
                for t in c.pages.values():
                    t[pages] = 50.0
                for d in c.slots.values():
                    for t in d.values():
                        t[slot] = 50
    assert all(at[k] == len(req[k]) for k in req) and gen.cache.num_free() == 9 and gen.cache.can_admit()
    for k in req:
        assert worst(torch.cat(got[k]), oracle("mixed", req[k]), limits("mixed", req[k], dtype)) < 1, k


@gpu
def test_pages_behind_the_widest_chunk_are_given_back():
    cfg, m = built("mixed")
    toks = tokens(300, cfg["vocab"], 6)
    gen = generator(m, blocks=4, max_seqs=1)                 # two chunks of 70 never need more
    got = feed(gen, gen.new_seq(), toks, [60, 2, 64, 1, 1, 30])
    assert worst(got, oracle("mixed", toks), limits("mixed", toks, torch.float32)) < 1
    assert gen.cache.live_blocks(0) <= 3 and gen.cache.num_free() >= 1


@gpu
@pytest.mark.parametrize("dtype,graphs", [(torch.float32, True), (torch.float32, False), (torch.bfloat16, True)])
def test_long_decoding_in_a_batch(dtype, graphs):
    """Three requests decode 170 tokens together (captured steps or eager), crossing page borders and chunk edges at different steps."""
    cfg, m = built("mixed", dtype)
    gen = generator(m, blocks=16, max_seqs=3, cuda_graphs=graphs)
    req = [tokens(n, cfg["vocab"], 20 + n) for n in (180, 233, 171)]
    seqs = [gen.new_seq() for _ in req]
    gen.prefill(seqs, [r[:len(r) - 170] for r in req])
    got = [gen.step(seqs, [[r[len(r) - 170 + i]] for r in req]).cpu() for i in range(170)]
    assert (gen._graphed is not None) == graphs
    for j, r in enumerate(req):
        assert worst(torch.stack([g[j] for g in got]), oracle("mixed", r)[-170:], limits("mixed", r, dtype)[-170:]) < 1


@gpu
def test_captures_survive_discarded_graphs():
    """A graph that becomes garbage (in a reference cycle) while another one is captured is freed behind the capture."""
    import gc
    from pmetal_b200.utils.graphs import capture

    class Owner:
        pass

    x = torch.ones(4, device="cuda")
    torch.cuda.synchronize()
    old = Owner()
    old.graph, old.self = torch.cuda.CUDAGraph(), old
    with capture(old.graph):
        x + 1
    new = torch.cuda.CUDAGraph()
    with capture(new):
        del old
        [[] for _ in range(200000)]                          # enough objects for several automatic collections
        y = x * 3
    assert gc.isenabled()
    new.replay()
    gc.collect()
    assert y.tolist() == [3.0] * 4


def _greedy(name, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(O.forward(seq, weights64(name), MODELS[name])[0][-1].argmax()))
    return seq[len(prompt):]


@gpu
@pytest.mark.parametrize("name", ["mixed", "ones"])
def test_greedy_generation_through_the_engine(name):
    """More requests than slots; prompts longer than a prefill portion run beside decoding slots in one batch."""
    from pmetal_b200.models.generation import Generator
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    cfg, m = built(name)
    prompts = [tokens(n, cfg["vocab"], 30 + n) for n in (5, 70, 1, 33, 90)]
    want = [_greedy(name, p, 8) for p in prompts]
    e = ContinuousBatchEngine(m, max_slots=2, num_blocks=8, prefill_chunk=31)
    mixed = []
    step = e.gen.step
    e.gen.step = lambda s, t, w=None: mixed.append([len(x) for x in t]) or step(s, t, w)
    reqs = [e.submit(Request(p, SamplingParams.greedy(8))) for p in prompts]
    while not all(r.done.is_set() for r in reqs):
        assert e.tick()
    assert [r.output for r in reqs] == want and any(len(x) == 2 and max(x) > 1 for x in mixed)
    assert e.cache.num_free() == 8
    g = Generator(m, cache=m.new_cache(16, max_seqs=6))
    res = g.generate(prompts[:2], SamplingParams.greedy(8), num_return_sequences=3)      # forks copy states, rings and latest tokens
    assert res.tokens == [want[0]] * 3 + [want[1]] * 3
    assert list(g.stream(prompts[3], SamplingParams.greedy(8))) == want[3]
    assert g.cache.num_free() == 16


@gpu
def test_generation_stops_at_the_last_position():
    from pmetal_b200.models.generation import Generator
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    _, m = built("ones")
    e = ContinuousBatchEngine(m, max_slots=2, num_blocks=16)
    r = e.generate(tokens(415, 40, 3), SamplingParams.greedy(50))
    assert r.finish_reason == "length" and len(r.output) == 6      # the token behind the last position is sampled, not read
    late = e.submit(Request(tokens(421, 40, 3), SamplingParams.greedy(2)))
    e.tick()
    assert late.finish_reason == "error:too_long"
    g = Generator(m, cache=m.new_cache(16, max_seqs=2))
    res = g.generate([tokens(415, 40, 3), tokens(20, 40, 4)], SamplingParams.greedy(12))
    assert res.tokens[0] == r.output and len(res.tokens[1]) == 12 and res.finish_reasons == ["length", "length"]
    assert list(g.stream(tokens(415, 40, 3), SamplingParams.greedy(12))) == r.output


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
    m = build_model(copy.deepcopy(PRESETS["ravapel-tiny"]), torch.float32, "cpu").init_weights(0.05, 3)
    save_pretrained(m, str(tmp_path))
    assert main(["infer", "-m", str(tmp_path), "-p", "hello", "--greedy", "--max-tokens", "5", "--json", "--kv-blocks", "16"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["generated_tokens"] == 5 and out["prompt_tokens"] == 5
    assert main(["infer", "-m", "random:ravapel-tiny", "-p", "hi", "--profile-layers", "--json"]) == 0
    assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["layers"]) == 6      # two of the four layers run twice
    data = tmp_path / "d.jsonl"
    data.write_text('{"text": "some words"}\n{"text": "and a few more"}\n')
    assert main(["eval", "-m", str(tmp_path), "-d", str(data)]) == 0
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["perplexity"] > 1


@gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(tmp_path, monkeypatch, capsys, dtype):
    """Steps on standard input, logits in files; the pool holds just what the live requests need."""
    import numpy as np
    from pmetal_b200.serve import trace
    cfg = MODELS["mixed"]
    m = build_model(cfg, torch.bfloat16, "cpu")
    m.load_hf_state_dict(weights16("mixed"))
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
    lx, ly, lz = (limits("mixed", t, getattr(torch, dtype)) for t in (x, y, z))
    assert worst(load(0), ox[[0, 98]], lx[[0, 98]]) < 1 and worst(load(1), ox[[99]], lx[[99]]) < 1
    assert worst(load(3), torch.cat([oz[[69, 3]], oy[[29]]]), torch.cat([lz[[69, 3]], ly[[29]]])) < 1
