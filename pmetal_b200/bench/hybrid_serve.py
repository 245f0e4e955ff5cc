"""Serving throughput of the hybrid decoder beside the closest other model at equal size, and its kernels beside the like
kernels of the other models (``bench.py --serve-hybrid``). Random weights; device time by CUDA events.

Duvivik and Ravapel presets stand beside the dense fast decoder (Ravapel's with one layer per layer run, its weights counted once per
run: equal work per token); Resevik presets beside the Qwen3-MoE decoder with the same width, experts
and attention heads and one layer per layer run (a looped stack has more runs than stored layers); Vosezen presets beside the same
with the layers' head counts of 128 channels and experts as wide as makes the stored weights equal (its experts have two matrices
and a shared one, the other's have three)."""
from __future__ import annotations

import math
import statistics
from typing import Callable, Dict, List

import torch

from ..models import hybrid_decoder as hd
from ..models.config import ModelArgs
from ..models.decoder import DecoderLM
from ..models.generation import Generator
from ..models.kv_cache import BLOCK, PagedKVCache
from ..models.mixers import RotationFreqs, StepContext
from ..models.state_cache import CacheSpec, StateCache, attention_runs, split_groups
from ..ops import native as nat
from ..utils.graphs import capture
from .kernels import peaks

# dense models of the fast path with about the same width, depth of weights and parameter count
DENSE = {
    "duvivik-1b": dict(hidden_size=2048, intermediate_size=6144, num_hidden_layers=12, num_attention_heads=16,
                       num_key_value_heads=8),
    "duvivik-2b": dict(hidden_size=2560, intermediate_size=9728, num_hidden_layers=19, num_attention_heads=32,
                       num_key_value_heads=8),
    "ravapel-1b": dict(hidden_size=2048, intermediate_size=7552, num_hidden_layers=18, num_attention_heads=16,
                       num_key_value_heads=4),
    "ravapel-2b": dict(hidden_size=2560, intermediate_size=9856, num_hidden_layers=28, num_attention_heads=20,
                       num_key_value_heads=4),
}


def like_kind(name: str) -> str:
    return "dense" if hd.PRESETS[name]["architecture"] in ("Duvivik", "Ravapel") else "moe"


def run_weights(args) -> int:
    """Matrix entries that one token meets in the layers and passes (weights of looped layers once per run)."""
    m = hd.HybridDecoderLM(args, torch.bfloat16, "meta")
    sizes = [sum(math.prod(s) for _, s, *_ in l.named_weights() if len(s) == 2) for l in m.layers]
    passes = sum(1 for _, again in m.runs if again) if m.loop_in is not None else 0
    return sum(sizes[i] for i, _ in m.runs) + passes * 2 * args.hidden_size ** 2


def like_expert_width(ex: dict) -> int:
    """Width of gated experts with as many weights as those of ``ex`` (a multiple of 128)."""
    if "shared" not in ex:
        return ex["expert"]["ff"]
    E = ex["router"]["experts"]
    return round(2 * (E * ex["expert"]["ff"] + ex["shared"]["ff"]) / (3 * E * 128)) * 128


def build(name: str, kind: str):
    args = hd.HybridArgs.from_dict(hd.PRESETS[name])
    if kind == "hybrid":
        return hd.HybridDecoderLM(args, torch.bfloat16, "cuda").init_weights(0.02, 0, "cuda").eval()
    if kind == "moe":
        from ..parallel.ep import shard_experts
        at = next(l["mixer"] for l in args.layers if l["type"] == "attention")
        ex = next(l["mlp"] for l in args.layers if l["mlp"])
        cfg = ModelArgs(vocab_size=args.vocab_size, hidden_size=args.hidden_size, num_hidden_layers=len(args.runs),
                        num_attention_heads=at["heads"], num_key_value_heads=at["kv_heads"], head_dim=128,
                        intermediate_size=like_expert_width(ex), moe_intermediate_size=like_expert_width(ex),
                        num_experts=ex["router"]["experts"], num_experts_per_tok=ex["router"]["top"],
                        tie_word_embeddings=args.design.tied)
        m = DecoderLM(cfg, torch.bfloat16, "cuda").init_weights_on_device().eval()
        for p in m.parameters():
            p.requires_grad_(False)
        m.size = sum(p.numel() for p in m.parameters())
        for layer in m.layers:
            shard_experts(layer.mlp, None, max_tokens=4096)
            layer.mlp.gate_up = torch.nn.Parameter(torch.empty(0, dtype=torch.bfloat16, device="cuda"), requires_grad=False)
            layer.mlp.down = torch.nn.Parameter(torch.empty(0, dtype=torch.bfloat16, device="cuda"), requires_grad=False)
        return m
    cfg = ModelArgs(vocab_size=args.vocab_size, head_dim=128, tie_word_embeddings=False, **DENSE[name])
    m = DecoderLM(cfg, torch.bfloat16, "cuda").init_weights_on_device().eval()
    for p in m.parameters():
        p.requires_grad_(False)
    return m


def event_ms(fn: Callable[[], None], iters: int) -> float:
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def throughput(model, context: int = 1024, prompt: int = 4096, batches=(1, 16, 64), steps: int = 48) -> Dict[str, dict]:
    """Prefill of one long prompt and of four prompts together; decode of several batch sizes from ``context`` tokens, token
    ids read back every step."""
    V = model.cfg.vocab_size
    g = torch.Generator().manual_seed(0)
    kw = {"max_seqs": max(batches)} if getattr(model, "slotted_cache", False) else {}
    gen = Generator(model, cache=model.new_cache(max(batches) * (-(-(context + steps + 16) // BLOCK) + 1) + 4 * prompt // BLOCK, **kw))
    out = {}
    for n_seq in (1, 4):
        prompts = [torch.randint(0, V, (prompt // n_seq,), generator=g).tolist() for _ in range(n_seq)]

        def run():
            seqs = [gen.new_seq() for _ in prompts]
            gen.prefill(seqs, prompts, chunk=prompt)
            for s in seqs:
                gen.cache.free_sequence(s)
        for _ in range(3):
            run()
        ms = event_ms(run, 5)
        out[f"prefill_{n_seq}x{prompt // n_seq}"] = {"ms": round(ms, 3), "tokens_per_s": round(prompt / ms * 1e3)}
    for n in batches:
        seqs = [gen.new_seq() for _ in range(n)]
        ids = gen.prefill(seqs, [torch.randint(0, V, (context,), generator=g).tolist() for _ in range(n)]).argmax(-1)

        def step():
            nonlocal ids
            ids = gen.decode_step(seqs, ids).argmax(-1)
            ids.tolist()
        for _ in range(8):
            step()
        ms = event_ms(step, steps)
        out[f"decode_b{n}"] = {"ms": round(ms, 4), "tokens_per_s": round(n / ms * 1e3, 1)}
        for s in seqs:
            gen.cache.free_sequence(s)
    nat.check_status()
    return out


def graph_us(fn: Callable[[], None], iters: int = 15) -> float:
    """Median device time of one captured call with a cold L2 (256 MB written before every replay)."""
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for _ in range(2):
            fn()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with capture(g):
        fn()
    ts = []
    for _ in range(iters + 3):
        flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        g.replay()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b) * 1e3)
    return statistics.median(ts[3:])


def _bf(*shape, scale=1.0):
    return (torch.randn(*shape, device="cuda") * scale).to(torch.bfloat16)


def _group(cache, n_seq: int, prior: int, new: int):
    """Batch in which ``n_seq`` sequences with ``prior`` cached tokens bring ``new`` each."""
    for i in range(n_seq):
        cache.add_sequence(i)
        if prior:
            cache.reserve(i, prior)
    meta = cache.prepare(list(range(n_seq)), [new] * n_seq)
    return meta, (split_groups(meta, 1 << 30)[0] if isinstance(cache, StateCache) else None)


def parallel_kernel_cases(name: str, batch: int = 16, ctx: int = 4096, prompt: int = 4096) -> List[dict]:
    """``kernel_cases`` for the parallel stacks (linear attention, windowed attention, experts with weighted inputs)."""
    from ..models.moe import WeightedInputExperts
    from ..parallel.ep import FusedExpertMoE
    cfg = hd.HybridArgs.from_dict(hd.PRESETS[name])
    W = cfg.hidden_size
    first = lambda kind: next(l["mixer"] for l in cfg.layers if l["type"] == kind)      # noqa: E731
    at, lin, ret = first("attention"), first("lightning"), first("retention")
    ex = next(l["mlp"] for l in cfg.layers if l["mlp"])
    E, k, ff = ex["router"]["experts"], ex["router"]["top"], ex["expert"]["ff"]
    H, G, D, win = at["heads"], at["kv_heads"], at["dim"], at["mask"]["size"]
    pk, out = peaks(), []

    def case(label, fn, nbytes=0, flops=0):
        us = graph_us(fn)
        bound = max(nbytes / pk["hbm_gbs"] / 1e3, flops / pk["bf16_tflops"] / 1e6)
        out.append({"kernel": label, "us": round(us, 2), "bound_us": round(bound, 2), "of_measured_peak": round(bound / us, 3)})

    f = lambda *s: torch.randn(*s, device="cuda")      # noqa: E731
    experts = WeightedInputExperts(ex, W, torch.bfloat16, "cuda")
    with torch.no_grad():
        for t in (experts.gate_up, experts.down):
            t.normal_(0.0, 0.02)
        experts.router.normal_(0.0, W ** -0.5)
    for mode, n_seq, prior, new in (("decode", batch, ctx - 1, 1), ("prefill", 1, 0, prompt)):
        T, blocks = n_seq * new, n_seq * (prior + new) // BLOCK + n_seq + 1
        tag = f"{mode} T={T} "
        # recurrences at the sizes of both linear layers | state-space recurrence of the same state
        for label, m, rot in (("lightning", lin, 0), ("retention", ret, ret["rot"]["dims"])):
            LH, N, P = m["heads"], m["dim"], m["vdim"]
            c = StateCache([CacheSpec(slots={"state": ((LH, N, P), torch.float32)})], blocks, n_seq, torch.bfloat16, "cuda")
            meta, grp = _group(c, n_seq, prior, new)
            u, y = _bf(T, 2 * LH * (N + P)), torch.empty(T, LH * P, dtype=torch.bfloat16, device="cuda")
            cs, sn = (f(T, rot // 2), f(T, rot // 2)) if rot else (None, None)
            dec = torch.full((LH,), 0.99, device="cuda")
            fn, d = (nat.linear_scan, dec) if mode == "decode" else (nat.linear_chunk, dec.log2())
            dims = (LH, N, P, rot, "half" if rot else "none", not rot)
            state_b = 2 * n_seq * LH * N * P * 4
            blk = 2 * T * LH * (64 * (N + P) / 2 + 2 * N * P) if mode == "prefill" else 0
            case(tag + label + " recurrence", lambda: fn(u, cs, sn, d, 1.0, c.slots[0]["state"], grp, dims, y),
                 T * LH * (2 * N + 2 * P) * 2 + state_b, blk)
        S = (LH, P, N, LH, 4)
        inner, conv = LH * P, LH * P + 2 * LH * N
        c = StateCache([CacheSpec(slots={"conv": ((4, conv), None), "state": ((LH, N, P), torch.float32)})], blocks, n_seq,
                       torch.bfloat16, "cuda")
        meta, grp = _group(c, n_seq, prior, new)
        us = _bf(T, -(-(inner + conv + LH) // 8) * 8)
        vec = (f(4, conv), f(conv), f(LH) - 3, f(LH), f(LH))
        sfn = nat.ssm_scan if mode == "decode" else nat.ssm_chunk
        case(tag + "  | ssm recurrence", lambda: sfn(us, *vec, c.slots[0]["conv"], c.slots[0]["state"], grp, S, y),
             T * (conv + inner + LH) * 2 + state_b, blk)
        nw = f(inner)
        gate = u[:, 2 * LH * N + inner:]
        case(tag + "norm of all heads + gate", lambda: nat.norm_gate(y, gate, nw, 1e-5, 1, False), 3 * T * inner * 2)
        case(tag + "norm per head + gate", lambda: nat.norm_gate(y, gate, None, 1e-5, LH, True), 3 * T * inner * 2)
        case(tag + "  | ssm gate + norm", lambda: nat.ssm_gate_norm(y, us, nw, 1e-5, 8, c.slots[0]["conv"], meta, S), 3 * T * inner * 2)
        # residual sum with the experts' rows
        x, yo, z, lw, h = f(T, W), _bf(T, W), _bf(T * k, W), f(W), _bf(T, W)
        inv = torch.randperm(T * k, device="cuda").int()
        case(tag + "sum of sublayers + rms norm", lambda: nat.add_rmsnorm(x, lw, 1e-5, y=yo, z=z, inv=inv, k=k, out=x),
             T * W * (4 + 2 + 2 * k + 4 + 2))
        rw = _bf(W)
        case(tag + "  | residual sum + rms norm", lambda: nat.rmsnorm_fwd(h, rw, 1e-6, yo), 4 * T * W * 2)
        # experts: routing, gather, both products (and the combination) | the same of the MoE decoder
        eng = FusedExpertMoE(experts.gate_up.data, experts.down.data, E, k, T)
        used = min(E, T * k)
        nb, fl = used * 3 * ff * W * 2 + 2 * T * k * (W + ff) * 2, 2 * T * k * 3 * ff * W
        case(tag + "router, routing and experts", lambda: experts(h), nb, fl)
        case(tag + "  | router, routing and experts", lambda: eng.forward(h, torch.nn.functional.linear(h, experts.router[:E])), nb, fl)
        del eng
        # windowed attention | paged attention in the same window
        c2 = StateCache([CacheSpec(page_width=2 * G * D)], blocks, n_seq, torch.bfloat16, "cuda")
        meta, grp = _group(c2, n_seq, prior, new)
        c2.pages[0].normal_()
        ua, rd = _bf(T, (H + G) * D), at["rot"]["dims"]
        cs, sn = f(T, rd // 2), f(T, rd // 2)
        prep = lambda: nat.window_prep(ua, cs, sn, (H, G, 1, D, D), (rd, "pairs"), True, 1e-5, (H * D, H * D), c2.pages[0], meta.slots)      # noqa: E731
        case(tag + "rotation + head norm + append", prep, T * (H + G) * D * 2 * 2 + T * G * D * 2)
        c3 = PagedKVCache(1, G, 128, blocks, device="cuda")
        meta3, _ = _group(c3, n_seq, prior, new)
        c3.k[0].normal_()
        c3.v[0].normal_()
        qkv, cs3, sn3, w128 = _bf(T, (H + 2 * G) * 128), f(T, 64), f(T, 64), _bf(128)
        case(tag + "  | rotation + head norm + append",
             lambda: nat.qknorm_rope_cache(qkv, w128, w128, cs3, sn3, H, G, 1e-6, c3.k[0], c3.v[0], meta3.slots),
             T * (2 * H + 4 * G) * 128 * 2)
        q, o = prep(), torch.empty(T, H * D, dtype=torch.bfloat16, device="cuda")
        if mode == "decode":
            pairs, keys = n_seq * min(win, ctx), n_seq * min(win, ctx)
        else:
            pairs, keys = sum(min(i + 1, win) for i in range(new)), 0
        case(tag + f"attention in a window of {win}",
             lambda: nat.window_attn(q, c2.pages[0], grp, (H, G, 1, D, D), win, 0.09, mode == "decode", o), keys * 2 * G * D * 2, pairs * H * 4 * D)
        q3 = _bf(T, H, 128)
        case(tag + "  | paged attention, same window", lambda: nat.paged_attn(q3, c3.k[0], c3.v[0], meta3, 0.09, win),
             keys * 2 * G * 128 * 2, pairs * H * 4 * 128)
        del c, c2, c3
        torch.cuda.empty_cache()
    nat.check_status()
    return out


def branch_kernel_cases(name: str, batch: int = 16, ctx: int = 4096, prompt: int = 4096) -> List[dict]:
    """``kernel_cases`` for the stacks with normed branches (latent attention with latent queries, difference and sink attention,
    experts with weighted outputs)."""
    from ..models.moe import WeightedOutputExperts
    from ..parallel.ep import FusedExpertMoE
    cfg = hd.HybridArgs.from_dict(hd.PRESETS[name])
    W = cfg.hidden_size
    first = lambda kind: next(l["mixer"] for l in cfg.layers if l["type"] == kind)      # noqa: E731
    at, df, sk = first("latent_attention"), first("attention"), first("attention_2")
    ex = next(l["mlp"] for l in cfg.layers if l["mlp"])
    E, I, k, ff, sf = ex["router"]["experts"], ex["router"]["identity"], ex["router"]["top"], ex["expert"]["ff"], ex["shared"]["ff"]
    pk, out = peaks(), []

    def case(label, fn, nbytes=0, flops=0):
        us = graph_us(fn)
        bound = max(nbytes / pk["hbm_gbs"] / 1e3, flops / pk["bf16_tflops"] / 1e6)
        out.append({"kernel": label, "us": round(us, 2), "bound_us": round(bound, 2), "of_measured_peak": round(bound / us, 3)})

    f = lambda *s: torch.randn(*s, device="cuda")      # noqa: E731
    experts = WeightedOutputExperts(ex, W, torch.bfloat16, "cuda")
    ffl = like_expert_width(ex)
    gu, dn = _bf(E, 2 * ffl, W, scale=0.02), _bf(E, W, ffl, scale=0.02)
    with torch.no_grad():
        for t in (experts.up, experts.down, experts.shared_up, experts.shared_down):
            t.normal_(0.0, 0.02)
        experts.router.normal_(0.0, W ** -0.5)
    for mode, n_seq, prior, new in (("decode", batch, ctx - 1, 1), ("prefill", 1, 0, prompt)):
        T, blocks = n_seq * new, n_seq * (prior + new) // BLOCK + n_seq + 1
        tag = f"{mode} T={T} "
        few = mode == "decode"
        pairs, keys = n_seq * (new * prior + new * (new + 1) // 2), n_seq * (prior + new)
        # latent attention: the query latent's norm beside the append, both projections of the queries | rotation, append
        H, dn_, dr, dv, r, qr = at["heads"], at["dim"], at["rot_dim"], at["vdim"], at["kv_rank"], at["q_rank"]
        row = -(-(r + dr) // 16) * 16
        dims = (H, dn_, dr, dv, r, row)
        c = StateCache([CacheSpec(page_width=row + 8)], blocks, n_seq, torch.bfloat16, "cuda")
        meta, grp = _group(c, n_seq, prior, new)
        c.pages[0].normal_()
        u, wukv, cs, sn = _bf(T, qr + r + dr), _bf(H * (dn_ + dv), r, scale=r ** -0.5), f(T, dr // 2), f(T, dr // 2)
        f_w = f(max(r, qr))
        qd, o, runs = _bf(T, H * (dn_ + dr)), torch.empty(T, H * dv, dtype=torch.bfloat16, device="cuda"), attention_runs(meta, grp)
        case(tag + "latent norms + rotation + append",
             lambda: nat.latent_prep(u, f_w[:r], 1e-5, cs, sn, dims, c.pages[0], meta.slots, qr, f_w[:qr]), T * 2 * (2 * qr + 2 * (r + dr)))if (f_w := f(max(r, qr))) is not None else None
        u1 = _bf(T, H * (dn_ + dr) + r + dr)
        case(tag + "  | latent norm + rotation + append", lambda: nat.latent_prep(u1, f_w[:r], 1e-5, cs, sn, dims, c.pages[0], meta.slots),
             T * 2 * (2 * H * dr + 2 * (r + dr)))
        if few:
            nb = keys * row * 2 + wukv.numel() * 2
            case(tag + f"latent attention with rotation, {ctx} keys",
                 lambda: nat.latent_attn(qd, wukv, wukv[H * dn_:], c.pages[0], grp, dims, 0.1, o, (cs, sn)), nb)
            case(tag + "  | latent attention", lambda: nat.latent_attn(qd, wukv, wukv[H * dn_:], c.pages[0], grp, dims, 0.1, o), nb)
        else:
            def latent():
                nat.latent_prep(qd, None, 1e-5, cs, sn, dims, None, meta.slots)
                nat.latent_expand_attn(qd, wukv, c.pages[0], runs[0], dims, 0.1, o)
            fl = pairs * H * 2 * (dn_ + dr + dv) + 2 * T * wukv.numel()
            case(tag + "rotation, latent attention, expanded", latent, 0, fl)
            case(tag + "  | latent attention, expanded", lambda: nat.latent_expand_attn(qd, wukv, c.pages[0], runs[0], dims, 0.1, o), 0, fl)
        del c
        # difference and sink attention | paged attention with as many heads of 128
        for label, m, M in (("difference", df, 2), ("sink", sk, 1)):
            H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            dims = (H, G, M, D, DV)
            c = StateCache([CacheSpec(page_width=G * (M * D + DV))], blocks, n_seq, torch.bfloat16, "cuda")
            meta, grp = _group(c, n_seq, prior, new)
            c.pages[0].normal_()
            runs = attention_runs(meta, grp)
            n_in = H * M * D + G * (M * D + DV) + H
            ua, wn = _bf(T, -(-n_in // 8) * 8), f(D)
            cols = (H * M * D, (H + G) * M * D)
            wide = 0 if few else nat.window_wide(dims, torch.bfloat16, 0)
            prep = lambda: nat.window_prep(ua, None, None, dims, (0, "none"), True, 1e-5, cols, c.pages[0], meta.slots, wn, wn, (0.3, 512),      # noqa: E731
                                           meta.positions, wide)
            case(tag + f"{label}: head norm + query factor + append", prep, 2 * T * (n_in - H) * 2)
            q, o = prep(), torch.empty(T, H * DV, dtype=torch.bfloat16, device="cuda")
            gate, lam, s = ua[:, n_in - H:], f(1), f(H)
            kw = dict(gate=gate, diff=(lam, 0.7, 1e-5)) if M == 2 else dict(gate=gate, softcap=50.0, sink=s)
            case(tag + f"{label} attention" + (f", {ctx} keys" if few else ""),
                 lambda: (nat.window_expand_attn(q, c.pages[0], grp, runs, dims, 0.09, o, **kw) if wide else
                          nat.window_attn(q, c.pages[0], grp, dims, 0, 0.09, few, o, **kw)),
                 keys * 2 * G * (M * D + DV) if few else 0, pairs * H * M * 2 * (D + DV))
            del c
            c3 = PagedKVCache(1, G, 128, blocks, device="cuda")
            meta3, _ = _group(c3, n_seq, prior, new)
            c3.k[0].normal_()
            c3.v[0].normal_()
            qkv, cs3, sn3, w128 = _bf(T, (H + 2 * G) * 128), f(T, 64), f(T, 64), _bf(128)
            case(tag + "  | head norm + rotation + append",
                 lambda: nat.qknorm_rope_cache(qkv, w128, w128, cs3, sn3, H, G, 1e-6, c3.k[0], c3.v[0], meta3.slots),
                 T * (2 * H + 4 * G) * 128 * 2)
            q3 = _bf(T, H, 128)
            case(tag + "  | paged attention", lambda: nat.paged_attn(q3, c3.k[0], c3.v[0], meta3, 0.09),
                 keys * 2 * G * 256 if few else 0, pairs * H * 4 * 128)
            del c3
        # sums
        x, y, zr, lw, h, rw = f(T, W), _bf(T, W), _bf(T * k, W), f(W), _bf(T, W), _bf(W)
        inv = torch.randperm(T * k, device="cuda").int()
        ids, wt = torch.randint(0, E + I, (T, k), device="cuda").int(), torch.rand(T, k, device="cuda")
        case(tag + "norm of a branch + sum", lambda: nat.add_normed(x, lw, 1e-6, y=y, w_base=1.0, out=x), T * W * (4 + 2 + 4 + 2))
        case(tag + "weighted rows + norm + sum", lambda: nat.add_normed(x, lw, 1e-6, y=y, z=zr, route=(wt, ids, inv, E), k=k, w_base=1.0, out=x),
             T * W * (4 + 2 + 2 * k + 4 + 2))
        case(tag + "  | residual sum + rms norm", lambda: nat.rmsnorm_fwd(h, rw, 1e-6, y), 4 * T * W * 2)
        # experts
        z, corr = f(T, E + I), f(E + I) * 0.01
        gr = ex["router"]["groups"]
        case(tag + "routing with grouped choice", lambda: nat.moe_route(z, k, False, choice=(corr, gr["count"], gr["keep"], 2.0)),
             T * (E + I + 4 * k) * 4)
        case(tag + "  | routing", lambda: nat.moe_route(z, k, True), T * (E + I + 4 * k) * 4)
        eng = FusedExpertMoE(gu, dn, E, k, T)
        live = E / (E + I)
        used = min(E, round(T * k * live))
        nb = used * 2 * ff * W * 2 + 2 * sf * W * 2 + 2 * T * (k + 1) * (W + ff) * 2
        case(tag + "router, routing, experts, shared expert", lambda: experts(h), nb, 2 * T * (k * live * 2 * ff + 2 * sf) * W)
        case(tag + "  | router, routing and experts", lambda: eng.forward(h, torch.nn.functional.linear(h, experts.router[:E])),
             min(E, T * k) * 3 * ffl * W * 2 + 2 * T * k * (W + ffl) * 2, 2 * T * k * 3 * ffl * W)
        del eng
        if not few:
            a = _bf(T * k, ff)
            case(tag + "gelu", lambda: nat.gelu(a, a), 2 * a.numel() * 2)
            b = _bf(T * k, 2 * ff)
            case(tag + "  | swiglu", lambda: nat.swiglu_fwd(b), 3 * a.numel() * 2)
        torch.cuda.empty_cache()
    nat.check_status()
    return out


def sandwich_kernel_cases(name: str, batch: int = 16, ctx: int = 4096, prompt: int = 4096) -> List[dict]:
    """``kernel_cases`` for the stacks with norms on both sides of the sublayers (channel gates, attention with sigmoid weights in
    chunks, matrix memory, input convolution)."""
    cfg = hd.HybridArgs.from_dict(hd.PRESETS[name])
    W = cfg.hidden_size
    gt = next(l["mixer"] for l in cfg.layers if l["type"] == "hgrn2")
    both = next(l["mixer"] for l in cfg.layers if l["type"] == "parallel")
    at, me = both["left"], both["right"]
    ff = next(l["mlp"]["ff"] for l in cfg.layers if l["mlp"])
    pk, out = peaks(), []

    def case(label, fn, nbytes=0, flops=0):
        us = graph_us(fn)
        bound = max(nbytes / pk["hbm_gbs"] / 1e3, flops / pk["bf16_tflops"] / 1e6)
        out.append({"kernel": label, "us": round(us, 2), "bound_us": round(bound, 2), "of_measured_peak": round(bound / us, 3)})

    f = lambda *s: torch.randn(*s, device="cuda")      # noqa: E731
    for mode, n_seq, prior, new in (("decode", batch, ctx - 1, 1), ("prefill", 1, 0, prompt)):
        T, blocks = n_seq * new, n_seq * (prior + new) // BLOCK + n_seq + 1
        tag = f"{mode} T={T} "
        few = mode == "decode"

        def cache(slots=None, page=0):
            c = StateCache([CacheSpec(page_width=page, slots=slots or {})], blocks, n_seq, torch.bfloat16, "cuda")
            return (c, *_group(c, n_seq, prior, new))
        # channel gates and matrix memory | the state-space recurrence with a state of the same size
        for label, m in (("channel gates", gt), ("matrix memory", me)):
            H, N, P = m["heads"], m["dim"], m["vdim"]
            c, meta, grp = cache({"state": ((H, N, P), torch.float32), "norm": ((H, N), torch.float32), "max": ((H, P // 4), torch.float32)})
            store = c.slots[0]
            y, den = torch.empty(T, H * P, dtype=torch.bfloat16, device="cuda"), torch.rand(T, H, device="cuda") + 0.5
            state_b = 2 * n_seq * H * N * P * 4
            blk = 0 if few else 2 * T * H * (64 * (N + P) / 2 + 2 * N * P)
            if label == "channel gates":
                u, z, b, lo = _bf(T, H * (N + P)), f(T, H * N) + 3, f(H * N), torch.rand(H * N, device="cuda")
                fn = nat.channel_scan if few else nat.channel_chunk
                case(tag + label + " recurrence", lambda: fn(u, u[:, H * N:], z, b, lo, store["state"], grp, (H, N, P), y),
                     T * H * ((N + 2 * P) * 2 + N * 4) + state_b, blk)
                w = f(P)
                case(tag + "norm per head", lambda: nat.norm_gate(y, None, w, 1e-5, H, False), 2 * T * H * P * 2)
            else:
                u, z, b, g = _bf(T, H * (2 * N + 2 * P)), f(T, 2 * H), f(2 * H) + 2, (10.0, N ** -0.5, 1e-6)
                v = u[:, 2 * H * N:]
                if few:
                    case(tag + label + " recurrence", lambda: nat.memory_scan(u, u[:, H * N:], v, z, b, g, store, grp, (H, N, P), y, den),
                         T * H * (2 * N + 2 * P) * 2 + state_b)
                else:
                    case(tag + label + " recurrence", lambda: nat.memory_chunk(u, 0, H * N, v, z, b, g, store, grp, (H, N, P), y, den),
                         T * H * (2 * N + 2 * P) * 2 + state_b, blk)
                w = f(H * P)
                case(tag + "normaliser + norm per head + gate", lambda: nat.norm_gate(y, u[:, H * (2 * N + P):], w, 1e-5, H, False, den), 3 * T * H * P * 2)
            S = (H, P, N, H, 4)
            inner, conv = H * P, H * P + 2 * H * N
            c2, meta, grp2 = cache({"conv": ((4, conv), None), "state": ((H, N, P), torch.float32)})
            us = _bf(T, -(-(inner + conv + H) // 8) * 8)
            vec = (f(4, conv), f(conv), f(H) - 3, f(H), f(H))
            sfn = nat.ssm_scan if few else nat.ssm_chunk
            case(tag + "  | ssm recurrence", lambda: sfn(us, *vec, c2.slots[0]["conv"], c2.slots[0]["state"], grp2, S, y),
                 T * (conv + inner + H) * 2 + state_b, blk)
            nw = f(inner)
            case(tag + "  | ssm gate + norm", lambda: nat.ssm_gate_norm(y, us, nw, 1e-5, H, c2.slots[0]["conv"], meta, S), 3 * T * inner * 2)
            del c, c2
        # attention with sigmoid weights in chunks | with a softmax in a window that sees as many keys on average
        H, G, D, DV, size = at["heads"], at["kv_heads"], at["dim"], at["vdim"], at["mask"]["size"]
        dims = (H, G, 1, D, DV)
        c, meta, grp = cache(page=G * (D + DV))
        c.pages[0].normal_()
        ua, rd, wn = _bf(T, H * D + G * (D + DV)), at["rot"]["dims"], f(D)
        cs, sn = f(T, rd // 2), f(T, rd // 2)
        prep = lambda: nat.window_prep(ua, cs, sn, dims, (rd, "half"), True, 1e-5, (H * D, H * D + G * D), c.pages[0], meta.slots, wn, wn,      # noqa: E731
                                       wide=0 if few else nat.window_wide(dims, torch.bfloat16, size, True))
        case(tag + "head norm + rotation + append", prep, 2 * T * (H * D + G * (D + DV)) * 2)
        c3 = PagedKVCache(1, G, 128, blocks, device="cuda")
        meta3, _ = _group(c3, n_seq, prior, new)
        c3.k[0].normal_()
        c3.v[0].normal_()
        qkv, cs3, sn3, w128 = _bf(T, (H + 2 * G) * 128), f(T, 64), f(T, 64), _bf(128)
        case(tag + "  | head norm + rotation + append",
             lambda: nat.qknorm_rope_cache(qkv, w128, w128, cs3, sn3, H, G, 1e-6, c3.k[0], c3.v[0], meta3.slots), T * (2 * H + 4 * G) * 128 * 2)
        q, o = prep(), torch.empty(T, H * DV, dtype=torch.bfloat16, device="cuda")
        if few:
            pairs = keys = n_seq * ((ctx - 1) % size + 1)
        else:
            pairs, keys = sum(i % size + 1 for i in range(new)), 0
        mixer = hd.MIXERS["sigmoid_attention"](at, cfg, 0, torch.bfloat16, "cuda")
        ctxt = StepContext(meta, RotationFreqs())
        case(tag + f"sigmoid attention in chunks of {size}", lambda: mixer.attend(q, c.pages[0], ctxt, None, o, 1.0),
             keys * G * (D + DV) * 2, pairs * H * 2 * (D + DV))
        case(tag + "  | softmax attention in a window, as many keys",
             lambda: nat.window_attn(q, c.pages[0], grp, dims, size if few else size // 2, 0.09, few, o), keys * G * (D + DV) * 2,
             n_seq * min(size, ctx) * H * 2 * (D + DV) if few else sum(min(i + 1, size // 2) for i in range(new)) * H * 2 * (D + DV))
        q3 = _bf(T, H, 128)
        case(tag + "  | paged attention, the same window", lambda: nat.paged_attn(q3, c3.k[0], c3.v[0], meta3, 0.09, size if few else size // 2),
             keys * G * 512, n_seq * min(size, ctx) * H * 512 if few else sum(min(i + 1, size // 2) for i in range(new)) * H * 512)
        del c, c3
        # sums and norms, convolution, embedding, feed-forward
        x, yo, lw, bias, xb, rw = f(T, W), _bf(T, W), f(W), f(W), _bf(T, W), _bf(W)
        c, meta, grp = cache({"canon": ((cfg.taps - 1, W), None), "token": ((1,), torch.int32)})
        taps, ring = f(cfg.taps, W), c.slots[0]["canon"]
        case(tag + "norm + sum + norm", lambda: nat.branch_norm(x, 1e-5, 1.0, y=yo, bias=bias, wb=lw, wn=lw, out=x), T * W * (4 + 2 + 4 + 2))
        if few:
            conv = (taps, ring, meta.state_slots, meta.positions)
            case(tag + "norm + sum + norm + convolution", lambda: nat.branch_norm(x, 1e-5, 1.0, y=yo, bias=bias, wb=lw, wn=lw, out=x, conv=conv),
                 T * W * (4 + 2 + 4 + 2 + 2 * cfg.taps) + cfg.taps * W * 4)
        else:
            case(tag + "input convolution", lambda: nat.canon(yo, taps, ring, meta), 2 * T * W * 2)
        case(tag + "  | residual sum + rms norm", lambda: nat.rmsnorm_fwd(xb, rw, 1e-6, yo), 4 * T * W * 2)
        ids, tab, pos = torch.randint(0, 30000, (T,), device="cuda"), _bf(30000, W), _bf(cfg.max_positions, W)
        case(tag + "embedding of pairs and positions", lambda: nat.pair_embed(ids, tab, tab, pos, meta, c.slots[0]["token"], (29999, 31, 5)),
             T * W * (3 * 2 + 4))
        case(tag + "  | embedding", lambda: nat.embed_scale(ids, tab, 1.0), T * W * (2 + 4 + 2))
        wgu, bgu = _bf(2 * ff, W, scale=W ** -0.5), f(2 * ff)
        if few:
            case(tag + "gate/up mat-vec with biases", lambda: nat.gemv_ex(xb, wgu, bgu, (float("inf"), 1.0, 0.0), n=ff), 2 * ff * W * 2)
            case(tag + "  | gate/up mat-vec, swiglu", lambda: nat.gemv(xb, wgu, swiglu=True), 2 * ff * W * 2)
        else:
            gu = _bf(T, 2 * ff)
            case(tag + "gated unit with biases", lambda: nat.clamped_glu(gu, ff, float("inf"), 1.0, 0.0, bgu), 3 * T * ff * 2)
            case(tag + "  | swiglu", lambda: nat.swiglu_fwd(gu), 3 * T * ff * 2)
        del c
        torch.cuda.empty_cache()
    nat.check_status()
    return out


def kernel_cases(name: str, batch: int = 16, ctx: int = 4096, prompt: int = 4096) -> List[dict]:
    """Every kernel of the hybrid layers at the sizes of preset ``name`` and, behind it, the like kernel of the other
    models: bytes and operations that the computation needs, device time, fraction of the slower of the two bounds."""
    cfg = hd.HybridArgs.from_dict(hd.PRESETS[name])
    W = cfg.hidden_size
    at = next(l["mixer"] for l in cfg.layers if l["type"] == "latent_attention")
    sm = next(l["mixer"] for l in cfg.layers if l["type"] == "mamba2")
    ff = next(l["mlp"]["ff"] for l in cfg.layers if l["mlp"])
    H, dn, dr, dv, r = at["heads"], at["dim"], at["rot_dim"], at["vdim"], at["kv_rank"]
    row = -(-(r + dr) // 16) * 16
    S = (sm["heads"], sm["vdim"], sm["state"], sm["groups"], sm["conv"])
    SH, P, N, G, taps = S
    inner, conv = SH * P, SH * P + 2 * G * N
    pk, out = peaks(), []

    def case(label, fn, nbytes=0, flops=0):
        us = graph_us(fn)
        bound = max(nbytes / pk["hbm_gbs"] / 1e3, flops / pk["bf16_tflops"] / 1e6)
        out.append({"kernel": label, "us": round(us, 2), "bound_us": round(bound, 2), "of_measured_peak": round(bound / us, 3)})

    f = lambda *s: torch.randn(*s, device="cuda")      # noqa: E731
    n_in = -(-(inner + conv + SH) // 8) * 8
    for mode, n_seq, prior, new in (("decode", batch, ctx - 1, 1), ("prefill", 1, 0, prompt)):
        T = n_seq * new
        tag = f"{mode} T={T} "
        # state-space recurrence (with its convolution) | gated delta rule scan
        c = StateCache([CacheSpec(slots={"conv": ((taps, conv), None), "state": ((SH, N, P), torch.float32)})],
                       n_seq * (prior + new) // BLOCK + n_seq + 1, n_seq, torch.bfloat16, "cuda")
        meta, grp = _group(c, n_seq, prior, new)
        u, y = _bf(T, n_in), torch.empty(T, inner, dtype=torch.bfloat16, device="cuda")
        vec = (f(taps, conv), f(conv), f(SH) - 3, f(SH), f(SH))
        fn = nat.ssm_scan if mode == "decode" else nat.ssm_chunk
        state_b = 2 * n_seq * SH * N * P * 4
        # products of the blocked form: scores and their use in the block, state in and out
        blk = 2 * T * SH * (64 * (N + P) / 2 + 2 * N * P) if mode == "prefill" else 0
        case(tag + "ssm recurrence", lambda: fn(u, *vec, c.slots[0]["conv"], c.slots[0]["state"], grp, S, y),
             T * (conv + inner + SH) * 2 + state_b, blk)
        gh = SH * N * P // (128 * 128)
        q, k, v = f(n_seq, new, gh, 128), f(n_seq, new, gh, 128), f(n_seq, new, gh, 128)
        gt, st = torch.rand(n_seq, new, gh, device="cuda"), f(n_seq, gh, 128, 128)
        yy = torch.empty_like(v)
        call = lambda: nat._chk(nat.lib().pm_gdn_scan(*[nat._p(t) for t in (q, k, v, gt, gt, st, yy)], nat.c_int(n_seq),      # noqa: E731
                                                      nat.c_int(new), nat.c_int(gh), nat.c_int(128), nat.c_int(128),
                                                      nat._stream()), "pm_gdn_scan")
        case(tag + "  | gated delta rule scan", call, 4 * T * gh * 128 * 4 + 2 * n_seq * gh * 128 * 128 * 4,
             2 * T * gh * (64 * 128 + 2 * 128 * 128) if mode == "prefill" else 0)
        # row kernels | rms norm, swiglu
        nw = f(inner)
        case(tag + "ssm gate + norm", lambda: nat.ssm_gate_norm(y, u, nw, 1e-5, sm["norm_groups"], c.slots[0]["conv"], meta, S),
             3 * T * inner * 2)
        x, yo, lw, lb = f(T, W), _bf(T, W), f(W), f(W)
        case(tag + "residual sum + layer norm", lambda: nat.post_layernorm(x, yo, lw, lb, 1e-5, 2.0), T * W * (4 + 2 + 4 + 2))
        xb, rw = _bf(T, W), _bf(W)
        case(tag + "  | residual sum + rms norm", lambda: nat.rmsnorm_fwd(xb, rw, 1e-6, yo), 4 * T * W * 2)
        wgu, bgu = _bf(2 * ff, W, scale=W ** -0.5), f(2 * ff)
        if mode == "decode":
            case(tag + "gate/up mat-vec, clamped", lambda: nat.gemv_ex(xb, wgu, bgu, (7.0, 1.702, 1.0), n=ff), 2 * ff * W * 2)
            case(tag + "  | gate/up mat-vec, swiglu", lambda: nat.gemv(xb, wgu, swiglu=True), 2 * ff * W * 2)
        else:
            gu = _bf(T, 2 * ff)
            case(tag + "clamped gated unit", lambda: nat.clamped_glu(gu, ff, 7.0, 1.702, 1.0, bgu), 3 * T * ff * 2)
            case(tag + "  | swiglu", lambda: nat.swiglu_fwd(gu), 3 * T * ff * 2)
        # attention | paged attention of the dense decoder at 16 / 8 heads of 128
        c2 = StateCache([CacheSpec(page_width=row + 8)], n_seq * (prior + new) // BLOCK + n_seq + 1, n_seq, torch.bfloat16, "cuda")
        meta, grp = _group(c2, n_seq, prior, new)
        c2.pages[0].normal_()
        dims = (H, dn, dr, dv, r, row)
        qd, wukv = _bf(T, H * (dn + dr) + r + dr), _bf(H * (dn + dv), r, scale=r ** -0.5)
        cs, sn = f(T, dr // 2), f(T, dr // 2)
        o = torch.empty(T, H * dv, dtype=torch.bfloat16, device="cuda")
        case(tag + "latent norm + rotation + append", lambda: nat.latent_prep(qd, nw[:r], 1e-5, cs, sn, dims, c2.pages[0], meta.slots),
             T * 2 * (2 * H * dr + 2 * (r + dr)))
        pairs = n_seq * (new * prior + new * (new + 1) // 2)
        if mode == "decode":
            case(tag + f"latent attention, {ctx} keys", lambda: nat.latent_attn(qd, wukv, wukv[H * dn:], c2.pages[0], grp, dims, 0.1, o),
                 n_seq * ctx * row * 2 + wukv.numel() * 2, pairs * H * 2 * (2 * r + dr))
        else:
            runs = attention_runs(meta, grp)
            case(tag + "latent attention, expanded", lambda: nat.latent_expand_attn(qd, wukv, c2.pages[0], runs[0], dims, 0.1, o),
                 0, pairs * H * 2 * (dn + dr + dv) + 2 * T * wukv.numel())
        c3 = PagedKVCache(1, 8, 128, n_seq * (prior + new) // BLOCK + n_seq + 1, device="cuda")
        meta3, _ = _group(c3, n_seq, prior, new)
        c3.k[0].normal_()
        c3.v[0].normal_()
        q3 = _bf(T, 16, 128)
        case(tag + "  | paged attention", lambda: nat.paged_attn(q3, c3.k[0], c3.v[0], meta3, 0.09),
             n_seq * (prior + new) * 8 * 128 * 4, pairs * 16 * 4 * 128)
        del c, c2, c3
        torch.cuda.empty_cache()
    nat.check_status()
    return out


def report(names: List[str], kernels: bool = True) -> dict:
    """Throughput of every named preset beside the closest other model of its size, and the kernel cases of the first."""
    res = {"what": "hybrid decoder beside the closest other model of equal size", "dtype": "bf16", "data": "synthetic",
           "device": torch.cuda.get_device_name(), "peaks": peaks(), "models": {}}
    for n in names:
        row = {}
        for kind in ("hybrid", like_kind(n)):
            m = build(n, kind)
            row[kind] = {"parameters": getattr(m, "size", None) or sum(p.numel() for p in m.parameters()), **throughput(m)}
            if kind == "hybrid" and m.loop_in is not None:
                row[kind]["weights_per_token"] = run_weights(m.cfg)
            del m
            torch.cuda.empty_cache()
        res["models"][n] = row
    if kernels:
        block = hd.HybridArgs.from_dict(hd.PRESETS[names[0]]).design.block
        cases = {"post": kernel_cases, "parallel": parallel_kernel_cases, "branch": branch_kernel_cases,
                 "sandwich": sandwich_kernel_cases}[block]
        res["kernels"] = {names[0]: cases(names[0])}
    return res
