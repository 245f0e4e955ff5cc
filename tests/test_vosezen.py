"""Vosezen on the hybrid decoder: kernels, mixers and experts against the plain statement in ``vosezen_oracle.py``, then whole
models through the generator's step function, the paged cache, the batching engine and the command line."""
import copy
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import vosezen_oracle as O
from test_hybrid_decoder import FP32, PORTIONS, err, feed, generator, tokens

from pmetal_b200.models.architectures import build_model, family_of
from pmetal_b200.models.hybrid_decoder import PRESETS, HybridArgs, HybridDecoderLM
from pmetal_b200.models.kv_cache import BLOCK
from pmetal_b200.models.loader import load_pretrained, save_pretrained
from pmetal_b200.models.moe import WeightedOutputExperts

gpu = pytest.mark.gpu


# ------------------------------------------------------------------------------------------- models of the tests
def latent(heads, dim, rot, vdim, rank, q_rank, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
            "scale": scale or 1.5 * (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot}}


def grouped(heads, kv, dim, vdim, temp=(0.4, 9), scale=None, **more):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.5 * dim ** -0.5,
            "q_temp": {"coef": temp[0], "every": temp[1]}, **more}


def difference(heads, kv, dim, vdim, diff, kv_from=None, **kw):
    return grouped(heads, kv, dim, vdim, diff=diff, **kw, **({} if kv_from is None else {"kv_from": kv_from}))


def sink(heads, kv, dim, vdim, softcap, **kw):
    return grouped(heads, kv, dim, vdim, softcap=softcap, **kw)


def kind(m):
    return "latent_attention" if "kv_rank" in m else ("attention" if "diff" in m else "attention_2")


def moe(ff, experts, identity, top, groups, shared, scale=1.7):
    m = {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
         "router": {"experts": experts, "identity": identity, "top": top, "scale": scale, "groups": dict(zip(("count", "keep"), groups))}}
    return m


def config(layers, width=48, vocab=101, eps=1e-5):
    """layers: (mixer, feed-forward or None)."""
    return {"architecture": "Vosezen", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": kind(m), "mixer": m, "mlp": f} for m, f in layers]}


MODELS = {
    # every mixer, keys and values of an earlier layer, one layer without feed-forward, choices in one, some and all groups
    "mixed": config([(sink(6, 2, 20, 28, 3.0), moe(40, 7, 2, 3, (3, 2), 24)), (latent(3, 24, 12, 20, 40, 56), moe(24, 5, 1, 1, (2, 1), 48)),
                     (difference(4, 2, 24, 40, 0.35), None), (difference(4, 2, 24, 40, 0.6, kv_from=2, temp=(0.9, 5)), moe(48, 8, 4, 4, (4, 2), 8)),
                     (latent(4, 16, 16, 32, 24, 32, base=300.0), moe(16, 4, 2, 6, (1, 1), 40)),
                     (sink(3, 3, 40, 16, 9.0, temp=(0.2, 64)), moe(32, 6, 0, 2, (3, 1), 16))]),
    # sizes that are not multiples of what the fast kernels copy at a time
    "odd": config([(difference(3, 1, 11, 7, 0.2), moe(33, 5, 1, 2, (2, 1), 13)), (latent(3, 7, 6, 5, 21, 11, base=37.0), moe(21, 3, 3, 2, (3, 2), 9)),
                   (sink(5, 5, 9, 22, 2.0, temp=(0.7, 3)), None), (difference(3, 1, 11, 7, 0.5, kv_from=0), moe(10, 4, 0, 1, (2, 2), 5))],
                  width=42, vocab=77, eps=1e-3),
    # everything that may be one or nothing
    "ones": config([(sink(1, 1, 1, 1, 1.0, temp=(1.0, 1)), moe(1, 1, 0, 1, (1, 1), 1)), (latent(1, 1, 2, 1, 1, 1), moe(8, 1, 1, 1, (1, 1), 8)),
                    (difference(1, 1, 8, 8, 0.0, temp=(0.0, 1)), None), (difference(2, 2, 1, 8, 0.9), moe(8, 2, 1, 1, (3, 1), 1, scale=1.0))],
                   width=32, vocab=40),
    # heads wider than the instances of the tensor-core kernels, many heads on one key, many experts and groups
    "wide": config([(difference(4, 2, 136, 72, 0.3), moe(64, 44, 4, 5, (8, 3), 96)), (sink(12, 1, 64, 264, 5.0), None),
                    (latent(20, 112, 32, 136, 72, 48), moe(72, 9, 3, 2, (6, 5), 8)), (difference(2, 1, 264, 24, 0.1), None),
                    (sink(4, 2, 200, 32, 8.0), moe(24, 3, 1, 3, (2, 2), 200)), (difference(12, 2, 64, 128, 0.5), None)], width=64, vocab=90),
}
CENTRES = 4


def _clear_choice(g, router, bound):
    """Logits of CENTRES kinds of token and a correction such that no choice of experts or groups is a close call. Corrections are
    negative on average: some of the chosen sums are below zero."""
    n = router["experts"] + router["identity"]
    for spread in (2.0, 3.0, 4.0, 5.0):
        for _ in range(400):
            lv = torch.randn(n, CENTRES, generator=g) * spread
            corr = torch.randn(n, generator=g) * 0.15 - 0.3
            s = torch.softmax(lv.t(), -1) + corr
            gap = choice_gap(s, router)
            if gap > bound:
                return lv, corr
    raise AssertionError("no clear routing found")


def choice_gap(s, router):
    """Smallest distance between the sums of a chosen and of a passed-over group or expert; s [tokens, outputs]."""
    count, keep, top, n = router["groups"]["count"], router["groups"]["keep"], router["top"], s.shape[1]
    best, at = s.reshape(-1, count, n // count).amax(-1).sort(-1, descending=True)
    gap = float((best[:, keep - 1] - best[:, keep]).min()) if keep < count else 9.0
    open_ = torch.zeros(s.shape[0], count).scatter(1, at[:, :keep], 1.0).repeat_interleave(n // count, 1) > 0
    c = s.masked_fill(~open_, -1e9).sort(-1, descending=True)[0]
    return min(gap, float((c[:, top - 1] - c[:, top]).min())) if top < n else gap


def random_weights(cfg, seed=0):
    """bf16-representable weights. Token vectors lie around a few centres and the routers tell the centres apart, so that
    rounding does not change which experts are chosen; sublayers add little to each sum, so that this holds in every layer."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    centres = torch.linalg.qr(torch.randn(W, CENTRES, generator=g))[0].t() * W ** 0.5
    routers = {}
    for i, l in enumerate(cfg["layers"]):
        if l["mlp"]:
            routers[i] = _clear_choice(g, l["mlp"]["router"], 0.12 if l["mlp"]["router"]["experts"] < 30 else 0.04)
    sd = {}
    for name, shape, _, _ in HybridDecoderLM(HybridArgs.from_dict(cfg), device="meta").named_weights():
        leaf = name.rsplit(".", 1)[-1]
        layer = int(name[1:].split(".")[0]) if name[0] == "l" else -1
        n = lambda s=1.0: torch.randn(shape, generator=g) * s      # noqa: E731
        if leaf == "router":
            t = routers[layer][0] @ centres / (3 * W)
        elif leaf == "correction":
            t = routers[layer][1]
        elif leaf in ("norm1", "norm2"):
            t = torch.rand(shape, generator=g) * 0.2 - 0.8
        elif name == "final.norm":
            t = torch.rand(shape, generator=g) * 0.4 - 0.2
        elif leaf == "norm":
            t = torch.rand(shape, generator=g) * 0.8 + 0.6
        elif leaf == "sink":
            t = n() + 1.0
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = n(0.7 * shape[0] ** -0.5)
        elif leaf == "embed":
            t = (centres[torch.arange(shape[0]) % CENTRES] + n(0.25)) * 3
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
    assert family_of(cfg) == "hybrid" and family_of({"model_type": "vosezen"}) == "hybrid"
    a = HybridArgs.from_dict(cfg)
    assert (a.vocab_size, a.hidden_size, a.num_hidden_layers, a.norm_eps, a.embed_scale) == (101, 48, 6, 1e-5, 1.0)
    assert a.to_hf_dict() == cfg and a.runs == [(i, False) for i in range(6)]
    m = build_model(cfg, torch.float32, "cpu")
    assert isinstance(m, HybridDecoderLM) and m.norm_b is None and m.head is m.embed_tokens
    names = [n for n, *_ in m.named_weights()]
    assert len(names) == len(set(names)) and "head" not in names
    assert not any(n.startswith("l3.mix.") and n.split(".")[2] in ("k", "v") for n in names)      # the layer reads layer 2's
    assert "l2.mlp.router" not in names and "l2.norm2" not in names and "l5.mlp.e5.down" in names and "l0.mlp.e7.up" not in names
    c = m.new_cache(4, max_seqs=2)
    assert sorted(c.pages) == [0, 1, 2, 4, 5] and not c.slots and c.can_truncate and c.window == 0
    assert c.pages[0].shape == (5, BLOCK, 2 * (24 + 32)) and c.pages[2].shape == (5, BLOCK, 2 * (2 * 24 + 40))
    assert c.pages[1].shape == (5, BLOCK, 64 + 8)
    with pytest.raises(RuntimeError, match="CUDA"):
        m(torch.tensor([1, 2]))


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "key/value"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "q_temp"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=2.5), "q_temp"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][2]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(dim=20), "must equal"),
    (lambda c: c["layers"][3]["mixer"].update(kv_heads=1), "must equal"),
    (lambda c: c["layers"][1]["mixer"].update(q_rank=0), "q_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "rot"),
    (lambda c: c["layers"][0].update(type="lightning"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=10), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=2), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=0), "groups"),
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
        lam = O.difference_factor(weights64("odd"), "l3.mix.", cfg["layers"][3]["mixer"])
        assert abs(float(back.layers[3].mixer.lam) - float(lam)) < 1e-6
    with pytest.raises(KeyError, match="l0.mlp.shared.up"):
        m.load_hf_state_dict({k: v for k, v in sd.items() if k != "l0.mlp.shared.up"})
    with pytest.raises(ValueError, match="shape"):
        m.load_hf_state_dict(dict(sd, **{"l1.mix.dq.norm": torch.zeros(4)}))


def test_engine_and_presets_build():
    from pmetal_b200 import build
    from pmetal_b200.serve.engine import ContinuousBatchEngine, Request
    m = build_model(MODELS["ones"], torch.float32, "cpu")
    e = ContinuousBatchEngine(m, max_slots=3, num_blocks=64)
    assert e.mixed and e.prefix is not None
    for _ in range(5):
        e.submit(Request([1, 2, 3]))
    e._admit()
    assert len(e.slots) == 3
    for p in ("vosezen-tiny", "vosezen-1b", "vosezen-2b"):
        HybridDecoderLM(HybridArgs.from_dict(PRESETS[p]), torch.bfloat16, "meta")
    a, args, d = load_pretrained("random:vosezen-tiny", torch.float32)
    assert d is None and args.model_type == "vosezen" and float(a.embed_tokens.abs().sum()) > 0
    assert float(a.norm_w.abs().sum()) == 0 and float(a.layers[1].mixer.q_norm_w.min()) == 1      # norms around zero and around one
    assert all(os.path.exists(os.path.join(build.CSRC, s + ".cu")) for s in build.COMPONENTS["vosezen"])


def _mix_entries(change):
    """cfg with ``change(mixer entry)`` applied to a copy of every mixer entry that has what is changed."""
    def run(cfg):
        c = copy.deepcopy(cfg)
        for l in c["layers"]:
            change(l["mixer"])
        return c
    return run


def _router_entries(change):
    def run(cfg):
        c = copy.deepcopy(cfg)
        for l in c["layers"]:
            if l["mlp"]:
                change(l["mlp"])
        return c
    return run


def _drop(key):
    return lambda m: m.pop(key, None)


def _route_with(monkeypatch, fn):
    """``fn(s, choice, allowed, router)`` -> (choice, weights' scores) replaces the end of the routing."""
    def route(h, w, correction, router):
        s = torch.softmax(h @ w.t(), -1)
        choice = s + correction
        n, count = choice.shape[1], router["groups"]["count"]
        best = choice.reshape(-1, count, n // count).amax(-1)
        kept = torch.argsort(best, dim=-1, descending=True, stable=True)[:, :router["groups"]["keep"]]
        allowed = torch.zeros_like(best, dtype=torch.bool).scatter(1, kept, True).repeat_interleave(n // count, 1)
        choice, ws = fn(s, choice, allowed, router)
        ids = torch.argsort(choice, dim=-1, descending=True, stable=True)[:, :router["top"]]
        return ids, ws.gather(1, ids) * router["scale"]
    monkeypatch.setattr(O, "route", route)


def _planted(monkeypatch, what, cfg):
    """Makes one mistake in the oracle; returns the configuration to run it with."""
    inf = float("-inf")
    real_diff, real_kv, real_q = O.difference_attention, O.keys_values, O.queries
    if what == "no cap":
        return _mix_entries(_drop("softcap"))(cfg)
    if what == "no temperature":
        return _mix_entries(_drop("q_temp"))(cfg)
    if what == "temperature one position late":
        real = O.temperature
        monkeypatch.setattr(O, "temperature", lambda T, m: torch.cat([real(1, m), real(T, m)[:-1]]))
    elif what == "no sink":
        real = O.attend
        monkeypatch.setattr(O, "attend", lambda q, k, v, scale, softcap=None, sink=None: real(q, k, v, scale, softcap))
    elif what == "sink capped":
        real = O.attend
        monkeypatch.setattr(O, "attend", lambda q, k, v, scale, softcap=None, sink=None: real(
            q, k, v, scale, softcap, None if sink is None else softcap * torch.tanh(sink / softcap)))
    elif what == "no gate":
        monkeypatch.setattr(O, "gated_output", lambda o, h, p, pre: O.linear(o.reshape(o.shape[0], -1), p[pre + "o"]))
    elif what == "one map":
        monkeypatch.setattr(O, "difference_factor", lambda p, pre, m: torch.zeros((), dtype=torch.float64))
    elif what == "lambda without its offset":
        real = O.difference_factor
        monkeypatch.setattr(O, "difference_factor", lambda p, pre, m: real(p, pre, m) - m["diff"])
    elif what == "maps interleaved":
        def kv(h, p, pre, m, eps, maps):
            k, v = real_kv(h, p, pre, m, eps, maps)
            return k.flip(2), v
        monkeypatch.setattr(O, "keys_values", kv)
    elif what == "key of the wrong group":
        def kv(h, p, pre, m, eps, maps):
            k, v = real_kv(h, p, pre, m, eps, maps)
            return k.roll(1, 1), v
        monkeypatch.setattr(O, "keys_values", kv)
    elif what == "no weight on the query norm":
        monkeypatch.setattr(O, "queries", lambda h, p, pre, m, eps, maps: real_q(h, dict(p, **{pre + "q.norm": torch.ones(m["dim"])}), pre, m, eps, maps))
    elif what == "one-plus weight on the key norm":
        monkeypatch.setattr(O, "keys_values", lambda h, p, pre, m, eps, maps: real_kv(h, dict(p, **{pre + "k.norm": 1 + p[pre + "k.norm"]}), pre, m, eps, maps))
    elif what == "keys of the layer's own input":
        monkeypatch.setattr(O, "difference_attention", lambda h, p, pre, m, eps, kv: real_diff(
            h, p, pre, m, eps, kv if m.get("kv_from") is None else O.keys_values(h, p, f"l{m['kv_from']}.mix.", m, eps, 2)))
    elif what == "no norm of the query latent":
        real = O.latent_attention
        def lat(h, p, pre, m, eps):
            unit, calls = O.unit_rms, []
            def skip(x, e):
                calls.append(1)
                return x if len(calls) == 1 else unit(x, e)
            O.unit_rms = skip
            try:
                return real(h, p, pre, m, eps)
            finally:
                O.unit_rms = unit
        monkeypatch.setattr(O, "latent_attention", lat)
    elif what == "halves rotated":
        def rot(x, base):
            d = x.shape[-1]
            order = torch.arange(d).view(2, -1).t().reshape(-1)
            y = torch.empty_like(x)
            y[..., order] = real_rot(x[..., order], base)
            return y
        real_rot = O.rotate_pairs
        monkeypatch.setattr(O, "rotate_pairs", rot)
    elif what == "norm weight without one":
        monkeypatch.setattr(O, "centred_norm", lambda x, w, eps: O.unit_rms(x, eps) * w)
    elif what == "no correction":
        _route_with(monkeypatch, lambda s, c, ok, r: (s.masked_fill(~ok, inf), s))
    elif what == "corrected weights":
        _route_with(monkeypatch, lambda s, c, ok, r: (c.masked_fill(~ok, inf), c))
    elif what == "zero for closed groups":
        _route_with(monkeypatch, lambda s, c, ok, r: (c.masked_fill(~ok, 0.0), s))
    elif what == "no groups":
        _route_with(monkeypatch, lambda s, c, ok, r: (c, s))
    elif what == "weights renormalised":
        real = O.route
        def route(h, w, corr, r):
            ids, ws = real(h, w, corr, r)
            return ids, ws / ws.sum(-1, keepdim=True)
        monkeypatch.setattr(O, "route", route)
    elif what == "no factor":
        return _router_entries(lambda m: m["router"].update(scale=1.0))(cfg)
    elif what == "no shared expert":
        return _router_entries(_drop("shared"))(cfg)
    elif what == "identities add nothing":
        real = O.mixture
        def mixture(h, p, pre, m):
            ids, ws = O.route(h, p[pre + "router"], p[pre + "correction"], m["router"])
            return real(h, p, pre, m) - (ws * (ids >= m["router"]["experts"])).sum(1, keepdim=True) * h
        monkeypatch.setattr(O, "mixture", mixture)
    return cfg


FAULTS = ["no cap", "no temperature", "temperature one position late", "no sink", "sink capped", "no gate", "one map",
          "lambda without its offset", "maps interleaved", "key of the wrong group", "no weight on the query norm",
          "one-plus weight on the key norm", "keys of the layer's own input", "no norm of the query latent", "halves rotated",
          "norm weight without one", "no correction", "corrected weights", "zero for closed groups", "no groups",
          "weights renormalised", "no factor", "no shared expert", "identities add nothing"]


@pytest.mark.parametrize("what", FAULTS)
def test_faults_show_in_the_test_model(monkeypatch, what):
    """The model the comparisons below use makes each of these mistakes visible: well above the fp32 tolerance, and above the bf16
    tolerance where the mistake is not a matter of rounding size."""
    toks = tokens(150, 101, 5)
    want, tol = oracle("mixed", toks), bound("mixed", toks, torch.bfloat16)
    cfg = _planted(monkeypatch, what, MODELS["mixed"])
    bad = err(O.forward(toks, weights64("mixed"), cfg)[0], want)
    assert bad > (30 * FP32 if what in ("sink capped", "temperature one position late") else 1.5 * tol), bad


def test_routers_of_the_test_models_decide_clearly(monkeypatch):
    """Rounding to bf16 does not change the chosen experts of any layer."""
    real, gaps = O.route, []

    def watch(h, w, correction, router):
        gaps.append(choice_gap((torch.softmax(h @ w.t(), -1) + correction).float(), router))
        return real(h, w, correction, router)
    monkeypatch.setattr(O, "route", watch)
    for name, cfg in MODELS.items():
        O.forward(tokens(60, cfg["vocab"], 5), weights64(name), cfg)
    assert min(gaps) > 0.01, gaps


def test_sequences_join_one_attention_launch():
    """A launch takes in fresh prompts whose rows follow; earlier tokens of its first sequence shift the queries against the keys."""
    from pmetal_b200.models.state_cache import CacheSpec, StateCache, attention_runs, split_groups
    c = StateCache([CacheSpec(page_width=8)], 16, 8, torch.float32, "cpu")
    for i in range(6):
        c.add_sequence(i)
    c.prepare([0], [70])
    c.prepare([4], [5])
    meta = c.prepare([0, 1, 2, 3, 4, 5], [30, 40, 1, 25, 20, 90])      # sequence 2 is a short portion, 4 has earlier tokens
    runs = attention_runs(meta, split_groups(meta, 16)[1])
    assert [(r.rows.start, r.rows.stop, r.n, r.shift) for r in runs] == [(0, 70, 70, 70), (71, 96, 25, 0), (96, 206, 110, 5)]
    at = lambda i, p: c.seqs[i].blocks[p // BLOCK] * BLOCK + p % BLOCK      # noqa: E731
    assert runs[0].slots.tolist() == [at(0, p) for p in range(100)] + [at(1, p) for p in range(40)]
    assert runs[2].slots.tolist() == [at(4, p) for p in range(25)] + [at(5, p) for p in range(90)]
    assert runs[0].seq_start.tolist() == [0] * 30 + [100] * 40 and runs[2].seq_start.tolist() == [0] * 20 + [25] * 90
    for r in runs:                                            # the last key row a query sees is its own
        rows = torch.arange(r.n) + r.shift
        assert torch.equal(r.slots[rows], meta.slots[r.rows])


# ------------------------------------------------------------------------------------------- kernels and modules
@gpu
@pytest.mark.parametrize("T,n,K", [(17, 1, 32), (64, 14, 192), (333, 33, 1024), (4100, 64, 96), (20, 20, 2048)])
def test_router_logits(T, n, K):
    from pmetal_b200.ops import functional as ops
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(T)
    h, w = torch.randn(T, K + 8, generator=g).to(torch.bfloat16), torch.randn(-(-n // 8) * 8, K, generator=g).to(torch.bfloat16)
    before = nat.LAUNCHES
    got = ops.router_logits(h.cuda()[:, :K], w.cuda(), n)
    assert nat.LAUNCHES == before + 1 and got.shape == (T, n) and got.dtype == torch.float32
    want = h[:, :K].double() @ w[:n].double().t()
    assert float((got.cpu().double() - want).abs().max()) < 1e-5 * K ** 0.5 * 4


@gpu
@pytest.mark.parametrize("cap", [0.0, 0.7, 30.0, 3000.0])
def test_flash_attention_with_cap_sink_and_gate(cap):
    """The tcgen05 kernel against the plain softmax: queries at an offset, documents, capped scores, a sink, output gates."""
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(int(cap))
    H, G, T, prior = 4, 2, 300, 70
    q, k, v = (torch.randn(n, h, 128, generator=g).to(torch.bfloat16) for n, h in ((T, H), (T + prior, G), (T + prior, G)))
    sink_, gate = torch.randn(H, generator=g) * 2 + 2, torch.randn(T, H + 4, generator=g).to(torch.bfloat16)
    start = torch.tensor([0] * 110 + [180] * 190, dtype=torch.int32)
    o, lse = nat.attn_fwd_rect(q.cuda(), k.cuda(), v.cuda(), start.cuda(), 0.12, prior, softcap=cap, sink=sink_.cuda(), gate=gate.cuda()[:, 4:])
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(H // G, 1)) * 0.12
    s = cap * torch.tanh(s / cap) if cap else s
    j, i = torch.arange(T + prior)[None], torch.arange(T)[:, None]
    s = s.masked_fill((j > i + prior) | (j < start[:, None]), float("-inf"))
    s = torch.cat([s, sink_.double()[:, None, None].expand(H, T, 1)], 2)
    want = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1)[:, :, :-1], v.double().repeat_interleave(H // G, 1))
    want = want * torch.sigmoid(gate.double()[:, 4:])[:, :, None]
    assert float((o.cpu().double() - want).abs().max()) < 0.02 * float(want.abs().max())
    torch.testing.assert_close(lse.cpu().double(), torch.logsumexp(s, -1), atol=2e-3, rtol=1e-3)
    nat.check_status()


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [48, 42, 1000, 2560])
def test_branch_norm_and_sum_kernel(dtype, width):
    """x + norm(y + weighted rows + weighted x), in place and not, with and without the routed part."""
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    n, k, E = 9, 3, 5
    x, w = r(n, width) * 3, r(width) * 0.3
    ybuf, z = r(n, width + 8).to(dtype), r(40, width).to(dtype)
    ids, wt = torch.randint(0, E + 2, (n, k), generator=g).int(), torch.rand(n, k, generator=g) * 2
    row = torch.randint(0, 40, (n, k), generator=g).int()
    row[ids >= E] = -7                                       # never read
    y = ybuf.cuda()[:, :width]
    take = torch.where((ids < E)[:, :, None], z.double()[row.clamp_min(0).long()], x.double()[:, None, :])
    routed = (wt.double()[:, :, None] * take).sum(1)
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)
    for with_y, with_route, base in ((True, True, 1.0), (False, True, 0.0), (True, False, 1.0)):
        s = (ybuf[:, :width].double() if with_y else 0) + (routed if with_route else 0)
        want = x.double() + O.unit_rms(s, 1e-3) * (base + w.double())
        xs = x.cuda()
        kw = dict(z=z.cuda(), route=(wt.cuda(), ids.cuda(), row.cuda(), E), k=k) if with_route else {}
        of, oc = nat.add_normed(xs, w.cuda(), 1e-3, y=y if with_y else None, w_base=base, out=xs if with_y else None, dtype=dtype, **kw)
        assert (of is xs) == with_y and oc.dtype == dtype
        torch.testing.assert_close(of.cpu().double(), want, rtol=2e-5, atol=2e-5)
        torch.testing.assert_close(oc.cpu().double(), want, **tol)
    rows = torch.tensor([8, 0, 3])
    _, oc = nat.add_rmsnorm(x.cuda(), w.cuda(), 1e-3, rows=rows.cuda(), dtype=dtype, want_stream=False, w_base=1.0)
    torch.testing.assert_close(oc.cpu().double(), O.centred_norm(x.double()[rows], w.double(), 1e-3), **tol)


@gpu
def test_exact_gelu():
    """The erf form, also far in the tails, as a kernel of its own and behind a mat-vec."""
    from pmetal_b200.ops import native as nat
    x = torch.cat([torch.linspace(-9, 9, 4001), torch.tensor([0.0, -30.0, 30.0])])
    x = torch.nn.functional.pad(x, (0, -len(x) % 24)).view(-1, 24)
    want = O.gelu(x.double())
    assert float((torch.nn.functional.gelu(x, approximate="tanh").double() - want).abs().max()) > 1e-4
    got = nat.gelu(x.cuda()).cpu().double()
    assert float((got - want).abs().max()) < 1e-6
    wide = torch.full((x.shape[0], 40), 5.0)
    wide[:, :17] = x[:, :17]
    v = wide.cuda()
    nat.gelu(v[:, :17], v[:, :17])
    assert float((v[:, :17].cpu().double() - want[:, :17]).abs().max()) < 1e-6 and bool((v[:, 17:] == 5).all())
    h = x.to(torch.bfloat16).cuda()
    assert float((nat.gelu(h).cpu().double() - O.gelu(h.cpu().double())).abs().max()) < 0.04
    w = torch.eye(24, dtype=torch.bfloat16, device="cuda")
    y = nat.gemv_ex(h[:11].contiguous(), w, out_f32=True, gelu=True).cpu().double()
    assert float((y - O.gelu(h[:11].cpu().double())).abs().max()) < 1e-6


ROUTERS = [dict(experts=14, identity=1, top=4, groups=(3, 2)), dict(experts=1, identity=0, top=1, groups=(1, 1)),
           dict(experts=6, identity=6, top=7, groups=(4, 3)), dict(experts=60, identity=4, top=16, groups=(32, 8)),
           dict(experts=90, identity=6, top=5, groups=(4, 1)), dict(experts=300, identity=20, top=6, groups=(8, 4)),
           dict(experts=3, identity=5, top=8, groups=(2, 2))]


@gpu
@pytest.mark.parametrize("T", [1, 37, 300, 1500])
@pytest.mark.parametrize("r", ROUTERS, ids=lambda r: f"{r['experts']}+{r['identity']}in{r['groups'][0]}")
def test_grouped_choice(r, T):
    """Choices, weights and the sorted order against the oracle; sums of score and correction on both sides of zero."""
    from pmetal_b200.ops import native as nat
    n, k = r["experts"] + r["identity"], r["top"]
    g = torch.Generator().manual_seed(n + T)
    z, corr = torch.randn(T, n + 5, generator=g) * 3, torch.randn(n, generator=g) * 0.3 - 0.2
    router = dict(r, scale=1.6, groups=dict(zip(("count", "keep"), r["groups"])))
    got = nat.moe_route(z.cuda()[:, :n], k, False, choice=(corr.cuda(), *r["groups"], 1.6))
    s = torch.softmax(z[:, :n].double(), -1)
    clear = torch.tensor([choice_gap((s[t:t + 1] + corr).float(), router) > 1e-5 for t in range(T)])
    assert float(clear.float().mean()) > 0.8
    ids, ws = O.route(z[:, :n].double(), torch.eye(n, dtype=torch.float64), corr.double(), router)
    order = torch.argsort(s + corr, dim=-1, descending=True)[:, :k]
    assert T < 300 or r["groups"][0] == r["groups"][1] or bool((order.sort(-1)[0] != ids.sort(-1)[0]).any())      # the groups matter
    assert torch.equal(got["topk_idx"].cpu().long()[clear], ids[clear])
    torch.testing.assert_close(got["topk_w"].cpu().double()[clear], ws[clear], rtol=1e-5, atol=1e-7)
    perm, inv, off = got["perm"].cpu().long(), got["inv"].cpu().long(), got["offsets"].cpu()
    assert torch.equal(perm[inv], torch.arange(T * k)) and off[-1] == T * k
    e = got["topk_idx"].cpu().flatten()[perm]
    assert torch.equal(e, e.sort()[0]) and torch.equal(off.diff(), torch.bincount(e, minlength=n).int())


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,experts,identity,top,groups,shared", [
    (64, 96, 6, 2, 3, (4, 2), 40), (48, 8, 1, 0, 1, (1, 1), 8), (42, 33, 5, 1, 3, (2, 1), 13), (64, 24, 40, 8, 4, (6, 3), 200),
    (128, 256, 3, 1, 1, (2, 1), 64), (64, 72, 4, 4, 5, (2, 2), 24), (64, 48, 2, 6, 2, (4, 2), 0)])
def test_experts_with_weighted_outputs(dtype, width, ff, experts, identity, top, groups, shared):
    """From one token to more rows than a tile per expert (mat-vecs, narrow tiles, padded slabs, row kernel); experts without
    rows, tokens that chose identities alone, no shared expert."""
    from pmetal_b200.ops import native as nat
    g = torch.Generator().manual_seed(ff)
    m = moe(ff, experts, identity, top, groups, shared)
    if not shared:
        del m["shared"]
    WeightedOutputExperts.check(m, 0)
    mod = WeightedOutputExperts(m, width, dtype, "cuda")
    p = {}
    with torch.no_grad():
        for name, shape, put, get in mod.named_weights():
            s = 0.1 if name == "correction" else (1.5 if name == "router" else 1.8) * shape[-1] ** -0.5
            p["m." + name] = (torch.randn(shape, generator=g) * s).to(torch.bfloat16)
            put(p["m." + name])
            assert torch.equal(get().cpu().to(torch.bfloat16), p["m." + name])
    p = {n: t.double() for n, t in p.items()}
    for n in (1, 2, 7, 16, 40, 333, 900):
        h = torch.randn(6 * n, width, generator=g).to(dtype)
        s = torch.softmax(h.double() @ p["m.router"].t(), -1) + p["m.correction"]
        clear = torch.tensor([choice_gap(s[t:t + 1].float(), m["router"]) > 0.004 for t in range(6 * n)])     # no close call
        h = h[clear][:n]
        x, w = h.float().cuda(), torch.zeros(width, device="cuda")
        got, _ = nat.add_normed(x, w, 1e-5, **mod(h.cuda()), w_base=1.0, dtype=dtype)
        run = lambda: O.unit_rms(O.mixture(h.double(), p, "m.", m), 1e-5)      # noqa: E731
        assert err(got.cpu().double() - h.double(), run()) < (bf16_bound(run, run()) if dtype == torch.bfloat16 else 1e-5), n
    nat.check_status()


def _mixer(m, width, dtype, seed, sd=None):
    cfg = config([(m, None)], width=width)
    sd = sd or random_weights(cfg, seed)
    model = build_model(cfg, dtype, "cuda")
    model.load_hf_state_dict(sd, strict=False)
    return model.layers[0].mixer, {k: v.double() for k, v in sd.items()}, model


def _run_mixer(mix, model, h, sizes):
    """h [T, width] through the mixer in portions; the sequence sits in shuffled pages, which hold what an earlier owner may have
    left."""
    from pmetal_b200.models.mixers import StepContext
    cache = model.new_cache(40, max_seqs=3)
    cache.free = [b for b in range(0, 40, 2)] + [b for b in range(1, 40, 2)]
    cache.add_sequence(0)
    cache.add_sequence(1)
    for t in cache.pages.values():
        t.fill_(7.0)
        if hasattr(mix, "q_rank"):
            t[..., mix.dims[4] + mix.dims[2]:] = 0           # pad columns are never written
    out, at, k = [], 0, 0
    while at < h.shape[0]:
        n = min(sizes[min(k, len(sizes) - 1)], h.shape[0] - at)
        meta = cache.prepare([1], [n])
        out.append(mix(h[at:at + n].contiguous(), cache, StepContext(meta, model._freqs), 0)[:, :h.shape[1]])
        at, k = at + n, k + 1
    return torch.cat(out)


def _id(m):
    return f"{kind(m)[-8:]}-h{m['heads']}d{m['dim']}v{m['vdim']}" + (f"q{m['q_rank']}r{m['kv_rank']}" if "q_rank" in m else f"g{m['kv_heads']}")


def _oracle_mixer(m, h, p):
    return O.mixer(kind(m), 0, h, p, m, 1e-5, {})


GROUPED = [difference(4, 2, 24, 40, 0.35), difference(3, 1, 11, 7, 0.2), difference(1, 1, 8, 8, 0.0), difference(12, 2, 64, 128, 0.5),
           difference(2, 2, 72, 24, 0.8), difference(2, 1, 136, 256, 0.3), difference(10, 1, 16, 16, 0.1), difference(2, 1, 264, 40, 0.1),
           difference(2, 1, 256, 192, 0.4), difference(2, 1, 24, 300, 0.4, scale=0.6), dict(difference(4, 4, 32, 96, 0.3), softcap=2.0),
           sink(6, 2, 20, 28, 3.0), sink(5, 5, 9, 22, 2.0), sink(1, 1, 1, 1, 1.0), sink(8, 2, 96, 96, 4.0), sink(20, 1, 64, 80, 30.0),
           sink(4, 2, 200, 32, 8.0), sink(12, 1, 64, 264, 5.0), sink(2, 2, 600, 8, 5.0), sink(3, 3, 40, 16, 0.5, temp=(3.0, 1)),
           sink(4, 1, 48, 128, 1e4)]


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", GROUPED, ids=_id)
def test_grouped_attention_mixers(dtype, m):
    mix, p, model = _mixer(m, 48, dtype, 1)
    h = torch.randn(200, 48, generator=torch.Generator().manual_seed(4)).to(dtype)
    run = lambda: _oracle_mixer(m, h.double(), p)      # noqa: E731
    want = run()
    single = _oracle_mixer(m, h.float(), {k: v.float() for k, v in p.items()})      # a_1 - lambda a_2 may cancel
    tol = bf16_bound(run, want) if dtype == torch.bfloat16 else max(FP32, 6 * err(single, want))
    for sizes in PORTIONS:
        assert err(_run_mixer(mix, model, h.cuda(), sizes), want) < tol, sizes


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m", [latent(3, 24, 12, 20, 40, 56), latent(3, 7, 6, 5, 21, 11, base=37.0), latent(1, 1, 2, 1, 1, 1),
                               latent(4, 16, 16, 32, 24, 32), latent(20, 96, 32, 128, 136, 72), latent(20, 112, 32, 136, 72, 48),
                               latent(2, 40, 8, 24, 512, 200), latent(17, 64, 64, 64, 256, 264, base=1e6)], ids=_id)
def test_latent_attention_with_latent_queries(dtype, m):
    mix, p, model = _mixer(m, 48, dtype, 1)
    h = torch.randn(200, 48, generator=torch.Generator().manual_seed(2)).to(dtype)
    run = lambda: _oracle_mixer(m, h.double(), p)      # noqa: E731
    want = run()
    single = _oracle_mixer(m, h.float(), {k: v.float() for k, v in p.items()})
    tol = bf16_bound(run, want) if dtype == torch.bfloat16 else max(FP32, 6 * err(single, want))
    for sizes in PORTIONS:
        assert err(_run_mixer(mix, model, h.cuda(), sizes), want) < tol, sizes


def _standout(what, D, T, dtype):
    """(mixer entry, weights, inputs, distance that each query asks for): a token vector is [what it asks for | what it is | its
    value]; keys are sign vectors, so that one score stands far above the others."""
    g = torch.Generator().manual_seed(1)
    W = 3 * D
    eye = lambda at: torch.eye(W)[at * D:(at + 1) * D]      # noqa: E731
    out = torch.zeros(W, D)
    out[:D] = torch.eye(D)
    one = torch.ones(D)
    if what == "latent":
        m = latent(1, D, 2, D, 2 * D, D, scale=0.6)
        dkv = torch.cat([eye(1), eye(2), torch.zeros(2, W)])
        first, second = torch.eye(2 * D)[:D], torch.eye(2 * D)[D:]
        uq = torch.cat([torch.eye(D), torch.zeros(2, D)])
        p = {"dq": eye(0), "dq.norm": one, "uq": uq, "dkv": dkv, "dkv.norm": torch.ones(2 * D), "uk": first, "uv": second, "o": out}
    elif what == "sink":
        m = sink(1, 1, D, D, 40.0, scale=0.4, temp=(0.5, 64))
        p = {"q": eye(0), "k": eye(1), "v": eye(2), "q.norm": one, "k.norm": one, "sink": torch.tensor([8.0]), "g": torch.zeros(1, W), "o": out}
    else:                                                    # the second map asks for the token itself
        m = difference(1, 1, D, D, 0.25, scale=0.4, temp=(0.5, 64))
        z = torch.zeros(D)
        p = {"q": torch.cat([eye(0), eye(1)]), "k": torch.cat([eye(1), eye(1)]), "v": eye(2), "q.norm": one, "k.norm": one, "lq1": z,
             "lk1": z, "lq2": z, "lk2": z, "g": torch.zeros(1, W), "o": out}
    keys, values = torch.randn(T, D, generator=g).sign(), torch.randn(T, D, generator=g)
    back = [0, 1, 63, 64, 65, 127, 128, 129, 2, 300]
    dist = torch.tensor([back[i % len(back)] if back[i % len(back)] <= i else (i if i % 2 else i // 2) for i in range(T)])
    h = torch.cat([keys[torch.arange(T) - dist], keys, values], 1).to(dtype)
    return m, {"l0.mix." + k: v.to(torch.bfloat16) for k, v in p.items()}, h


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("what", ["latent", "sink", "difference"])
def test_far_keys_and_page_borders(dtype, what):
    """Every query asks for one key: the token itself, neighbours, both sides of page borders, hundreds of tokens back, the first
    tokens. Asking for the next key instead changes the result altogether."""
    m, sd, h = _standout(what, 64, 420, dtype)
    mix, p, model = _mixer(m, 192, dtype, 0, sd)
    run = lambda x=h: _oracle_mixer(m, x.double(), p)[:, :64]      # noqa: E731
    want = run()
    off = torch.cat([h[1:, :64], h[:1, :64]])
    assert err(run(torch.cat([off, h[:, 64:]], 1)), want) > 0.5
    tol = bf16_bound(run, want) if dtype == torch.bfloat16 else FP32
    for sizes in ([420], [380, 1], [30, 2, 17, 64, 1, 90, 3], [1], [2], [64], [63, 1, 65]):
        assert err(_run_mixer(mix, model, h.cuda(), sizes)[:, :64], want) < tol, sizes


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_query_factor_steps_with_the_position(dtype):
    """Just before, at and behind the steps, at far positions, for intervals that do and do not divide page sizes."""
    from pmetal_b200.ops import native as nat
    pos = torch.tensor([0, 1, 5, 6, 7, 62, 63, 64, 126, 127, 128, 999, 1000, 1 << 20, (1 << 20) - 1], dtype=torch.int32)
    for D in (24, 11):
        u = torch.randn(len(pos), 3 * D, generator=torch.Generator().manual_seed(D)).to(dtype)
        for every in (1, 7, 64, 1000, 1 << 20):
            q = nat.window_prep(u.cuda(), None, None, (3, 1, 1, D, D), (0, "none"), True, 1e-5, (0, 0), None, None, None, None,
                                (0.7, every), pos.cuda())
            t = O.temperature(1 << 20, {"q_temp": {"coef": 0.7, "every": every}})[pos[:-2].long()] if every == 1 else None
            f = 1 + 0.7 * torch.log(((pos + 1) // every + 1).double())
            assert t is None or torch.allclose(t, f[:-2])
            want = O.unit_rms(u.double().view(-1, 3, D), 1e-5) * f[:, None, None]
            got = q.cpu().double()[:, :, :D]
            torch.testing.assert_close(got, want, **(dict(rtol=5e-3, atol=1e-6) if dtype == torch.bfloat16 else dict(rtol=2e-6, atol=1e-7)))


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
def test_stream_after_every_layer(name):
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
def test_mixed_batches_with_recycled_pages(dtype):
    """Four live requests of unequal lengths, portions beside single tokens, pauses, ends and new requests in used pages
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
                c, pages = gen.cache, gen.cache.seqs[seq[k]].blocks
                c.free_sequence(seq[k])
                for i, t in c.pages.items():
                    t[pages] = 50.0
                    mix = m.layers[i].mixer
                    if hasattr(mix, "q_rank"):
                        t[..., mix.dims[4] + mix.dims[2]:] = 0
    assert all(at[k] == len(req[k]) for k in req) and gen.cache.num_free() == 9 and gen.cache.can_admit()
    for k in req:
        assert err(torch.cat(got[k]), oracle("mixed", req[k])) < bound("mixed", req[k], dtype), k


@gpu
@pytest.mark.parametrize("dtype,graphs", [(torch.float32, True), (torch.float32, False), (torch.bfloat16, True)])
def test_long_decoding_in_a_batch(dtype, graphs):
    """Three requests decode 170 tokens together (captured steps or eager), crossing page borders at different steps."""
    cfg, m = built("mixed", dtype)
    gen = generator(m, blocks=16, max_seqs=3, cuda_graphs=graphs)
    req = [tokens(n, cfg["vocab"], 20 + n) for n in (180, 233, 171)]
    seqs = [gen.new_seq() for _ in req]
    gen.prefill(seqs, [r[:len(r) - 170] for r in req])
    got = [gen.step(seqs, [[r[len(r) - 170 + i]] for r in req]).cpu() for i in range(170)]
    assert (gen._graphed is not None) == graphs
    for j, r in enumerate(req):
        assert err(torch.stack([g[j] for g in got]), oracle("mixed", r)[-170:]) < bound("mixed", r, dtype)


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
    e = ContinuousBatchEngine(m, max_slots=2, num_blocks=8, prefill_chunk=31, prefix_cache=False)
    mixed = []
    step = e.gen.step
    e.gen.step = lambda s, t, w=None: mixed.append([len(x) for x in t]) or step(s, t, w)
    reqs = [e.submit(Request(p, SamplingParams.greedy(8))) for p in prompts]
    while not all(r.done.is_set() for r in reqs):
        assert e.tick()
    assert [r.output for r in reqs] == want and any(len(x) == 2 and max(x) > 1 for x in mixed)
    assert e.cache.num_free() == 8
    g = Generator(m, cache=m.new_cache(16, max_seqs=6))
    res = g.generate(prompts[:2], SamplingParams.greedy(8), num_return_sequences=3)      # forks share pages
    assert res.tokens == [want[0]] * 3 + [want[1]] * 3
    assert list(g.stream(prompts[3], SamplingParams.greedy(8))) == want[3]
    assert g.cache.num_free() == 16


@gpu
def test_prompt_prefixes_are_shared():
    """No recurrent layers: a second request forks the cached pages of the first one's prompt."""
    from pmetal_b200.models.sampling import SamplingParams
    from pmetal_b200.serve.engine import ContinuousBatchEngine
    cfg, m = built("mixed")
    e = ContinuousBatchEngine(m, max_slots=2, num_blocks=24)
    p = tokens(150, cfg["vocab"], 9)
    a = e.generate(p, SamplingParams.greedy(4))
    b = e.generate(p[:140] + [1, 2, 3], SamplingParams.greedy(4))
    assert e.stats.prefix_hits == 1 and b.cached_tokens == 128
    assert a.output == _greedy("mixed", p, 4) and b.output == _greedy("mixed", p[:140] + [1, 2, 3], 4)


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
    m = build_model(copy.deepcopy(PRESETS["vosezen-tiny"]), torch.float32, "cpu").init_weights(0.05, 3)
    save_pretrained(m, str(tmp_path))
    assert main(["infer", "-m", str(tmp_path), "-p", "hello", "--greedy", "--max-tokens", "5", "--json", "--kv-blocks", "16"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["generated_tokens"] == 5 and out["prompt_tokens"] == 5
    assert main(["infer", "-m", "random:vosezen-tiny", "-p", "hi", "--profile-layers", "--json"]) == 0
    assert len(json.loads(capsys.readouterr().out.strip().splitlines()[-1])["layers"]) == 5
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
    tol = max(bound("mixed", t, getattr(torch, dtype)) for t in (x, y, z))
    assert err(load(0), ox[[0, 98]]) < tol and err(load(1), ox[[99]]) < tol
    assert err(load(3), torch.cat([oz[[69, 3]], oy[[29]]])) < tol
