"""Config-driven serving decoder for stacks that mix kinds of attention and recurrent layers (Duvivik, Resevik, Vosezen, Ravapel).

Each layer has a token mixer (``mixers.MIXERS``) and optionally a feed-forward. The design (``DESIGNS``) says which mixers the
configuration's layer types mean and how the sublayers meet the stream:

* ``post``: both sublayers read the stream itself and the norm comes after the sum, x <- LN(alpha * x + sublayer(x));
* ``parallel``: both read one RMS norm of the stream, x <- x + mixer(h) + ff(h). A span of layers may run several times in a
  row with the same weights, every run with a cache or state of its own; each pass but the first starts by adding the
  embedding output to the stream. The sum, the re-added embedding and the next layer's norm are one kernel;
* ``branch``: both sublayers read the stream itself and only what they add is normed, x <- x + rms(sublayer(x)) (1 + w). The norm
  and the sum (for experts also the weighted sum of a token's rows) are one kernel;
* ``sandwich``: a norm before and one after every sublayer, x <- x + rms(sublayer(rms(x) (1 + w))) (1 + w'); the mixer's input gets a
  causal convolution over its own last values added. A span of layers may run several times; every pass starts with a projection of
  the stream beside the embedding output. The embedding adds a row chosen by the pair of the previous and the current token and a row of
  the position. Norm of the result, sum, norm of the next input and, in decode steps, the convolution are one kernel.

The stream, norms, rotation angles, softmax, routers and recurrent states are fp32; projections and their activations run in
the model's type (bf16 on the sm_100a kernels, or fp32 throughout with full-precision matrix products).

``forward_paged`` has the interface of ``DecoderLM.forward_paged``: the new tokens of several sequences in one batch, their
cache a ``StateCache``, so the generator, the CUDA-graph decoder, the continuous-batching engine and the sampler serve it
as they serve the other models. There is no CPU path: the model can be built, loaded and saved anywhere, and runs on a
GPU."""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..ops import functional as ops
from .kv_cache import BLOCK
from .mixers import MIXERS, RotationFreqs, StepContext, frozen
from .moe import WeightedInputExperts, WeightedOutputExperts
from .state_cache import CacheSpec, StateCache

GLU_BETA, GLU_SHIFT = 1.702, 1.0          # gate slope and the offset of the up half in the clamped gated unit



@dataclass(frozen=True)
class Design:
    block: str                            # "post", "parallel", "branch" or "sandwich"
    mixers: Dict[str, str]                # "type" of a layer -> name in MIXERS
    feed_forward: str                     # kind of the layers' "mlp" entries
    experts: Optional[type] = None        # class of the feed-forwards of kind "moe"
    tied: bool = False                    # the embedding table is the output projection
    norm_base: float = 0.0                # norms multiply with norm_base + weight ("branch", "sandwich")
    glu: Tuple[float, float] = (GLU_BETA, GLU_SHIFT)      # gate slope and offset of the up half of dense feed-forwards


DESIGNS: Dict[str, Design] = {
    "duvivik": Design("post", {"mamba2": "mamba2", "latent_attention": "latent_attention"}, "dense"),
    "resevik": Design("parallel", {"lightning": "lightning", "retention": "retention", "attention": "window_attention"}, "moe",
                      WeightedInputExperts),
    "vosezen": Design("branch", {"attention": "difference_attention", "latent_attention": "latent_attention",
                                 "attention_2": "sink_attention"}, "moe", WeightedOutputExperts, tied=True, norm_base=1.0),
    "ravapel": Design("sandwich", {"hgrn2": "channel_gate", "parallel": "sigmoid_attention_and_memory"}, "dense", norm_base=1.0,
                      glu=(1.0, 0.0)),
}


@dataclass
class HybridArgs:
    vocab_size: int
    hidden_size: int
    layers: List[dict]                    # {"type", "mixer", "mlp"} per layer, as in the configuration file
    embed_scale: float = 1.0
    residual_alpha: float = 1.0
    norm_eps: float = 1e-5
    model_type: str = "duvivik"
    loop: Optional[Tuple[int, int, int]] = None      # (first layer, layer behind the last, passes)
    pair: Optional[Tuple[int, int, int]] = None      # (buckets, factor of the previous id, factor of the id) of the pair embedding
    taps: int = 0                                    # of the mixers' input convolution
    max_positions: int = 0                           # rows of the position embedding; 0: sequences of any length
    bos_token_id: Optional[int] = None
    eos_token_id: Optional[int] = None
    raw: dict = field(default_factory=dict, repr=False)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def design(self) -> Design:
        return DESIGNS[self.model_type]

    @property
    def runs(self) -> List[Tuple[int, bool]]:
        """Layers in the order of execution: (layer, whether a further pass of the loop starts with it; in "sandwich" stacks, whether
        any pass does)."""
        n = len(self.layers)
        a, b, times = self.loop or (0, 0, 0)
        first = 0 if self.design.block == "sandwich" else 1
        order = [(i, False) for i in range(a)]
        for t in range(times):
            order += [(i, t >= first and i == a) for i in range(a, b)]
        return order + [(i, False) for i in range(b, n)]

    @classmethod
    def from_dict(cls, d: dict) -> "HybridArgs":
        name = str(d.get("architecture", d.get("model_type", ""))).lower()
        if name not in DESIGNS:
            raise ValueError(f"unknown hybrid architecture {name!r}")
        design = DESIGNS[name]
        layers = [dict(l, mlp=l.get("mlp")) for l in d["layers"]]
        for i, l in enumerate(layers):
            if l["type"] not in design.mixers:
                raise ValueError(f"layer {i}: unknown mixer {l['type']!r} (known: {', '.join(design.mixers)})")
            kind = MIXERS[design.mixers[l["type"]]]
            missing = [k for k in kind.KEYS if k not in l["mixer"]]
            if missing:
                raise ValueError(f"layer {i}: mixer entry lacks {', '.join(missing)}")
            kind.check(l["mixer"], i, layers)
            mlp = l["mlp"]
            if mlp is not None and mlp.get("kind") != design.feed_forward:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            if mlp is not None and design.experts is not None:
                design.experts.check(mlp, i)
        loop = d.get("loop")
        if loop is not None:
            loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if design.block not in ("parallel", "sandwich") or not 0 <= loop[0] < loop[1] <= len(layers) or loop[2] < 1:
                raise ValueError(f"loop {loop} over {len(layers)} layers")
        eos = d.get("eos_token_id")
        more = {}
        if design.block == "sandwich":
            e = d["embedding"]["bigram"]
            more = {"pair": (int(e["buckets"]), int(e["mul_prev"]), int(e["mul_cur"])), "taps": int(d["canon"]["taps"]),
                    "max_positions": int(d["max_positions"])}
            if more["pair"][0] < 1 or min(more["pair"]) < 0:
                raise ValueError(f"pair embedding with {e}")
            if not 1 <= more["taps"] <= 17:
                raise ValueError(f"input convolution of {more['taps']} taps (1 to 17 are built)")
            if more["max_positions"] < 1 or int(d["width"]) > 8192:
                raise ValueError("max_positions must be positive, width at most 8192")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   residual_alpha=float(d.get("postln_alpha", 1.0)), norm_eps=float(d["norm"]["eps"]), model_type=name, loop=loop,
                   bos_token_id=d.get("bos_token_id"), eos_token_id=eos[0] if isinstance(eos, list) else eos,
                   raw=copy.deepcopy(d), **more)

    @classmethod
    def from_pretrained(cls, model_dir: str) -> "HybridArgs":
        with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as fh:
            return cls.from_dict(json.load(fh))

    def to_hf_dict(self) -> dict:
        return copy.deepcopy(self.raw)


def _stack(width: int, vocab: int, ff: int, attn: dict, ssm: dict, pattern: str, limit: float = 7.0) -> dict:
    """Configuration dict: one letter per layer, A = latent attention with its own latents, a = reading those of the latest
    A, m = state-space layer without feed-forward, M = with one."""
    layers, src = [], None
    for i, ch in enumerate(pattern):
        mlp = {"kind": "dense", "ff": ff, "limit": limit} if ch in "AaM" else None
        if ch in "Aa":
            m = dict(attn)
            if ch == "A":
                src = i
            else:
                m["kv_from"] = src
            layers.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
        else:
            layers.append({"type": "mamba2", "mixer": dict(ssm), "mlp": mlp})
    return {"architecture": "Duvivik", "vocab": vocab, "width": width, "embedding": {"scale": 1.0}, "postln_alpha": 2.0,
            "norm": {"eps": 1e-5}, "layers": layers}


def _parallel_stack(width: int, vocab: int, ff: int, experts: int, top: int, linear: dict, attn: dict, pattern: str,
                    loop: Optional[Tuple[int, int, int]] = None) -> dict:
    """Configuration dict: one letter per layer, L = lightning, R = retention, A = windowed attention, all with experts."""
    h = linear["heads"]
    kinds = {"L": ("lightning", dict(linear, decay=[1.0 - 2.0 ** (-1.0 - 9.0 * i / max(h - 1, 1)) for i in range(h)])),
             "R": ("retention", dict(linear, decay=[1.0 - 2.0 ** (-5.0 - 5.0 * i / max(h - 1, 1)) for i in range(h)],
                                     rot={"base": 10000.0, "dims": linear["dim"]})),
             "A": ("attention", dict(attn))}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    d = {"architecture": "Resevik", "vocab": vocab, "width": width, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-5},
         "layers": [{"type": kinds[c][0], "mixer": copy.deepcopy(kinds[c][1]), "mlp": copy.deepcopy(mlp)} for c in pattern]}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


def _branch_stack(width: int, vocab: int, ff: int, shared: int, experts: int, identity: int, top: int, groups: Tuple[int, int],
                  latent: dict, diff: dict, sink: dict, pattern: str) -> dict:
    """Configuration dict: one letter per layer, L = latent attention, S = attention with a sink, D = difference attention, d = the
    same on the keys and values of the latest D; all with experts."""
    kinds = {"L": ("latent_attention", latent), "S": ("attention_2", sink), "D": ("attention", diff), "d": ("attention", diff)}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
           "router": {"experts": experts, "identity": identity, "top": top, "scale": 2.0,
                      "groups": dict(zip(("count", "keep"), groups))}}
    layers, src = [], None
    for i, c in enumerate(pattern):
        m = copy.deepcopy(kinds[c][1])
        if c == "D":
            src = i
        elif c == "d":
            m["kv_from"] = src
        layers.append({"type": kinds[c][0], "mixer": m, "mlp": copy.deepcopy(mlp)})
    return {"architecture": "Vosezen", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": layers}


def _sandwich_stack(width: int, vocab: int, ff: int, gate: dict, left: dict, right: dict, pattern: str, loop: Tuple[int, int, int],
                    positions: int = 8192) -> dict:
    """Configuration dict: one letter per layer, G = channel gates, P = attention and matrix memory side by side."""
    kinds = {"G": ("hgrn2", gate), "P": ("parallel", {"left": left, "right": right, "left_scale": 1.0, "right_scale": 0.8})}
    return {"architecture": "Ravapel", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": 1e-5},
            "embedding": {"bigram": {"buckets": 2 * vocab + 1, "mul_prev": 31, "mul_cur": 5}}, "canon": {"taps": 3},
            "loop": dict(zip(("start", "stop", "times"), loop)),
            "layers": [{"type": kinds[c][0], "mixer": copy.deepcopy(kinds[c][1]), "mlp": {"kind": "dense", "ff": ff}} for c in pattern]}


def _chunked(heads, kv_heads, dim, vdim, size, rot):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "mask": {"size": size},
            "rot": {"base": 10000.0, "dims": rot}}


def _memory(heads, dim, vdim, cap=10.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _grouped(heads, kv_heads, dim, vdim, every, **more):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5,
            "q_temp": {"coef": 0.2, "every": every}, **more}


def _linear(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def _window(heads, kv_heads, dim, size):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": size},
            "rot": {"base": 10000.0, "dims": dim // 2}}


def _attn(heads, dim, rot, vdim, rank):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": (dim + rot) ** -0.5,
            "rot": {"base": 10000.0, "dims": rot}}


def _q_latent(q_rank, *attn):
    return dict(_attn(*attn), q_rank=q_rank)


def _ssm(heads, vdim, state, groups, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


# random-weight models for smoke runs and measurements (``random:<name>``)
PRESETS: Dict[str, dict] = {
    "duvivik-tiny": _stack(64, 512, 96, _attn(4, 16, 8, 24, 40), _ssm(4, 24, 16, 2, norm_groups=2), "AmaM"),
    "duvivik-1b": _stack(2048, 65536, 6144, _attn(32, 64, 64, 128, 512), _ssm(64, 64, 128, 8, norm_groups=8), "Ammmammm" * 2),
    "duvivik-2b": _stack(2560, 65536, 9728, _attn(32, 96, 32, 128, 512), _ssm(80, 64, 128, 8, norm_groups=8), "Ammmammm" * 4),
    "resevik-tiny": _parallel_stack(64, 512, 48, 6, 2, _linear(3, 16, 24), _window(4, 2, 20, 40), "LRAL", (0, 3, 2)),
    # 12 layers twice, and 16 layers with the middle eight twice: 24 layer runs each
    "resevik-1b": _parallel_stack(1536, 65536, 768, 12, 2, _linear(12, 128, 96), _window(12, 4, 96, 512), "LRA" * 4, (0, 12, 2)),
    "resevik-2b": _parallel_stack(2048, 65536, 1024, 16, 2, _linear(16, 128, 128), _window(16, 8, 128, 1024), "LRAL" * 4, (4, 12, 2)),
    "vosezen-tiny": _branch_stack(64, 512, 48, 56, 7, 1, 2, (4, 2), _q_latent(40, 4, 16, 8, 24, 32), _grouped(4, 2, 16, 24, 32, diff=0.2),
                                  _grouped(6, 3, 24, 16, 48, softcap=30.0), "LSDLd"),
    "vosezen-1b": _branch_stack(1536, 65536, 768, 1536, 12, 4, 2, (4, 2), _q_latent(768, 16, 64, 32, 96, 256),
                                _grouped(12, 4, 64, 128, 1024, diff=0.3), _grouped(12, 4, 128, 128, 1024, softcap=50.0), "LSDLLSdL" * 2),
    "vosezen-2b": _branch_stack(2048, 65536, 1024, 2048, 16, 4, 2, (4, 2), _q_latent(1024, 16, 96, 32, 128, 512),
                                _grouped(16, 4, 64, 128, 1024, diff=0.3), _grouped(16, 4, 128, 128, 1024, softcap=50.0), "LSDLLSdL" * 3),
    "ravapel-tiny": _sandwich_stack(64, 512, 72, _linear(3, 16, 24), _chunked(4, 2, 20, 28, 40, 12), _memory(3, 24, 20), "GPPG", (1, 3, 2)),
    # 12 layers with the middle six twice (18 layer runs), and 20 layers with eight twice (28 layer runs)
    "ravapel-1b": _sandwich_stack(2048, 65536, 6144, _linear(16, 128, 128), _chunked(16, 4, 128, 128, 1024, 64), _memory(8, 128, 128),
                                  "GGP" * 4, (3, 9, 2)),
    "ravapel-2b": _sandwich_stack(2560, 65536, 8192, _linear(20, 128, 128), _chunked(20, 4, 128, 128, 1024, 64), _memory(10, 128, 128),
                                  "GPGG" * 5, (4, 12, 2)),
}


class ClampedMLP(nn.Module):
    """Gated feed-forward with biases on all projections: g sigmoid(beta g) (u + shift), g and u clamped where the entry has a
    ``limit``. ``glu`` = (beta, shift)."""

    def __init__(self, m: dict, width: int, dtype, device, glu: Tuple[float, float] = (GLU_BETA, GLU_SHIFT)):
        super().__init__()
        limit = m.get("limit")
        self.ff, self.width = m["ff"], width
        self.glu = (float("inf") if limit is None else float(limit), *glu)
        up8 = lambda n: -(-n // 8) * 8      # noqa: E731
        self.w_gu = frozen(torch.zeros(up8(2 * self.ff), width, dtype=dtype, device=device))
        self.b_gu = frozen(torch.zeros(2 * self.ff, device=device))
        self.w_down = frozen(torch.zeros(up8(width), self.ff, dtype=dtype, device=device))
        self.b_down = frozen(torch.zeros(width, device=device))

    def named_weights(self):
        f, w = self.ff, self.width
        yield "gate", (f, w), lambda t: self.w_gu[:f].copy_(t), lambda: self.w_gu[:f]
        yield "gate.b", (f,), lambda t: self.b_gu[:f].copy_(t), lambda: self.b_gu[:f]
        yield "up", (f, w), lambda t: self.w_gu[f:2 * f].copy_(t), lambda: self.w_gu[f:2 * f]
        yield "up.b", (f,), lambda t: self.b_gu[f:].copy_(t), lambda: self.b_gu[f:]
        yield "down", (w, f), lambda t: self.w_down[:w].copy_(t), lambda: self.w_down[:w]
        yield "down.b", (w,), self.b_down.copy_, lambda: self.b_down

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """Without the down-projection's bias, which the caller adds in fp32 with the residual."""
        from ..ops import native as nat
        glu = self.glu
        if x.dtype == torch.bfloat16 and ops.gemv_fits(*x.shape) and x.stride(0) % 8 == 0:
            a = nat.gemv_ex(x, self.w_gu, self.b_gu, glu, n=self.ff)
        else:
            a = nat.clamped_glu(ops.project(x, self.w_gu), self.ff, *glu, bias=self.b_gu)
        return ops.project(a, self.w_down)


class HybridLayer(nn.Module):
    def __init__(self, spec: dict, cfg: HybridArgs, index: int, dtype, device):
        super().__init__()
        self.cfg = cfg
        self.mixer = MIXERS[cfg.design.mixers[spec["type"]]](spec["mixer"], cfg, index, dtype, device)
        self.mlp = ClampedMLP(spec["mlp"], cfg.hidden_size, dtype, device, cfg.design.glu) if spec["mlp"] is not None else None
        vec = lambda: frozen(torch.zeros(cfg.hidden_size, device=device))      # noqa: E731
        self.norm1_w, self.norm1_b = vec(), vec()
        if self.mlp is not None:
            self.norm2_w, self.norm2_b = vec(), vec()

    def named_weights(self):
        vecs = [("norm1", self.norm1_w), ("norm1.b", self.norm1_b)]
        if self.mlp is not None:
            vecs += [("norm2", self.norm2_w), ("norm2.b", self.norm2_b)]
        for name, p in vecs:
            yield name, (self.cfg.hidden_size,), p.copy_, (lambda p=p: p)
        for pre, mod in (("mix.", self.mixer), ("mlp.", self.mlp)):
            if mod is not None:
                for name, *rest in mod.named_weights():
                    yield (pre + name, *rest)

    def forward(self, xf, xc, cache, ctx):
        """(fp32 stream, compute-type copy) -> the same after the layer."""
        from ..ops import native as nat
        cfg = self.cfg
        y = self.mixer(xc, cache, ctx)
        xf, xc = nat.post_layernorm(xf, y, self.norm1_w, self.norm1_b, cfg.norm_eps, cfg.residual_alpha)
        if self.mlp is not None:
            y = self.mlp(xc)
            xf, xc = nat.post_layernorm(xf, y, self.norm2_w, self.norm2_b, cfg.norm_eps, cfg.residual_alpha,
                                        bias=self.mlp.b_down)
        return xf, xc


class ParallelLayer(nn.Module):
    """One norm, read by the mixer and by the experts; the caller sums up (``HybridDecoderLM._parallel``)."""

    def __init__(self, spec: dict, cfg: HybridArgs, index: int, dtype, device):
        super().__init__()
        self.cfg = cfg
        self.mixer = MIXERS[cfg.design.mixers[spec["type"]]](spec["mixer"], cfg, index, dtype, device)
        self.mlp = cfg.design.experts(spec["mlp"], cfg.hidden_size, dtype, device) if spec["mlp"] is not None else None
        self.norm1_w = frozen(torch.zeros(cfg.hidden_size, device=device))

    def named_weights(self):
        yield "norm1", (self.cfg.hidden_size,), self.norm1_w.copy_, lambda: self.norm1_w
        for pre, mod in (("mix.", self.mixer), ("mlp.", self.mlp)):
            if mod is not None:
                for name, *rest in mod.named_weights():
                    yield (pre + name, *rest)

    def forward(self, h, cache, ctx, run):
        """(mixer output, expert rows, row of every (token, slot), experts per token)."""
        y = self.mixer(h, cache, ctx, run)
        return (y, *(self.mlp(h) if self.mlp is not None else (None, None, 1)))


class BranchLayer(nn.Module):
    """Sublayers read the stream and add their normed results to it."""

    def __init__(self, spec: dict, cfg: HybridArgs, index: int, dtype, device):
        super().__init__()
        self.cfg = cfg
        self.mixer = MIXERS[cfg.design.mixers[spec["type"]]](spec["mixer"], cfg, index, dtype, device)
        self.mlp = cfg.design.experts(spec["mlp"], cfg.hidden_size, dtype, device) if spec["mlp"] is not None else None
        self.norm1_w = frozen(torch.zeros(cfg.hidden_size, device=device))
        if self.mlp is not None:
            self.norm2_w = frozen(torch.zeros(cfg.hidden_size, device=device))

    def named_weights(self):
        for name, p in [("norm1", self.norm1_w)] + ([("norm2", self.norm2_w)] if self.mlp is not None else []):
            yield name, (self.cfg.hidden_size,), p.copy_, (lambda p=p: p)
        for pre, mod in (("mix.", self.mixer), ("mlp.", self.mlp)):
            if mod is not None:
                for name, *rest in mod.named_weights():
                    yield (pre + name, *rest)

    def forward(self, xf, xc, cache, ctx):
        """(fp32 stream, compute-type copy) -> the same after the layer."""
        from ..ops import native as nat
        cfg = self.cfg
        kw = dict(w_base=cfg.design.norm_base)
        xf, xc = nat.add_normed(xf, self.norm1_w, cfg.norm_eps, y=self.mixer(xc, cache, ctx), **kw)
        if self.mlp is not None:
            xf, xc = nat.add_normed(xf, self.norm2_w, cfg.norm_eps, **self.mlp(xc), **kw)
        return xf, xc


class SandwichLayer(nn.Module):
    """Norms before and after both sublayers and a convolution on the mixer's input; ``HybridDecoderLM._sandwich`` forms the first norm
    and the convolution, and adds what the last sublayer returns."""

    def __init__(self, spec: dict, cfg: HybridArgs, index: int, dtype, device):
        super().__init__()
        self.cfg = cfg
        self.mixer = MIXERS[cfg.design.mixers[spec["type"]]](spec["mixer"], cfg, index, dtype, device)
        self.mlp = ClampedMLP(spec["mlp"], cfg.hidden_size, dtype, device, cfg.design.glu) if spec["mlp"] is not None else None
        vec = lambda: frozen(torch.zeros(cfg.hidden_size, device=device))      # noqa: E731
        self.norm1_w, self.norm1b_w = vec(), vec()
        if self.mlp is not None:
            self.norm2_w, self.norm2b_w = vec(), vec()
        self.conv_w = frozen(torch.zeros(cfg.taps, cfg.hidden_size, device=device))      # [taps][channel]

    def cache_spec(self):
        spec = self.mixer.cache_spec()
        spec.slots["canon"] = ((self.cfg.taps - 1, self.cfg.hidden_size), None)
        return spec

    def named_weights(self):
        names = ("norm1", "norm1b") + (("norm2", "norm2b") if self.mlp is not None else ())
        for name in names:
            p = getattr(self, name + "_w")
            yield name, (self.cfg.hidden_size,), p.copy_, (lambda p=p: p)
        yield "canon1", (self.cfg.hidden_size, self.cfg.taps), lambda t: self.conv_w.copy_(t.t()), lambda: self.conv_w.t()
        for pre, mod in (("mix.", self.mixer), ("mlp.", self.mlp)):
            if mod is not None:
                for name, *rest in mod.named_weights():
                    yield (pre + name, *rest)

    def forward(self, x, h, cache, ctx, run):
        """(fp32 stream, mixer input) -> (stream, what is left to add to it: the last sublayer's result, its bias, the weight of the
        norm behind it)."""
        from ..ops import native as nat
        cfg = self.cfg
        last = {"y": self.mixer(h, cache, ctx, run), "wb": self.norm1b_w}
        if self.mlp is not None:
            x, h = nat.branch_norm(x, cfg.norm_eps, cfg.design.norm_base, wn=self.norm2_w, out=x, **last)
            last = {"y": self.mlp(h), "bias": self.mlp.b_down, "wb": self.norm2b_w}
        return x, last


class HybridDecoderLM(nn.Module):
    graph_decode = True         # single-token steps can be captured (generation.GraphedDecoder)
    mixed_batches = True        # the scheduler puts prompt portions and decoded tokens into one step
    slotted_cache = True        # ``new_cache`` takes the number of live sequences

    def __init__(self, cfg: HybridArgs, dtype=torch.float32, device=None):
        super().__init__()
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError("the hybrid decoder runs in bf16 or fp32")
        self.cfg, self.dtype = cfg, dtype
        self.embed_tokens = frozen(torch.zeros(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device))
        block = cfg.design.block
        kind = {"post": HybridLayer, "parallel": ParallelLayer, "branch": BranchLayer, "sandwich": SandwichLayer}[block]
        self.layers = nn.ModuleList([kind(s, cfg, i, dtype, device) for i, s in enumerate(cfg.layers)])
        self.runs = cfg.runs
        self.bigram = self.pos = self.loop_in = None
        if block == "sandwich":
            table = lambda n: frozen(torch.zeros(n, cfg.hidden_size, dtype=dtype, device=device))      # noqa: E731
            self.bigram, self.pos = table(cfg.pair[0] + 1), table(cfg.max_positions)
            if cfg.loop:
                self.loop_in = frozen(torch.zeros(-(-cfg.hidden_size // 8) * 8, 2 * cfg.hidden_size, dtype=dtype, device=device))
        self.norm_w = frozen(torch.zeros(cfg.hidden_size, device=device))
        self.norm_b = frozen(torch.zeros(cfg.hidden_size, device=device)) if block == "post" else None
        self.head = self.embed_tokens if cfg.design.tied else frozen(torch.zeros(cfg.vocab_size, cfg.hidden_size, dtype=dtype, device=device))
        self._freqs = RotationFreqs()

    # ------------------------------------------------------------------ weights
    def named_weights(self):
        """(checkpoint name, shape, setter, getter) of every tensor."""
        c = self.cfg
        yield "embed", (c.vocab_size, c.hidden_size), self.embed_tokens.copy_, lambda: self.embed_tokens
        for name in ("bigram", "pos"):
            p = getattr(self, name)
            if p is not None:
                yield name, tuple(p.shape), p.copy_, (lambda p=p: p)
        if self.loop_in is not None:
            w = c.hidden_size
            yield "loop.in", (w, 2 * w), lambda t: self.loop_in[:w].copy_(t), lambda: self.loop_in[:w]
        for i, layer in enumerate(self.layers):
            for name, *rest in layer.named_weights():
                yield (f"l{i}.{name}", *rest)
        yield "final.norm", (c.hidden_size,), self.norm_w.copy_, lambda: self.norm_w
        if self.norm_b is not None:
            yield "final.norm.b", (c.hidden_size,), self.norm_b.copy_, lambda: self.norm_b
        if not c.design.tied:
            yield "head", (c.vocab_size, c.hidden_size), self.head.copy_, lambda: self.head

    @torch.no_grad()
    def load_hf_state_dict(self, sd: Dict[str, torch.Tensor], strict: bool = True) -> List[str]:
        """Copy checkpoint tensors into place; returns the names that were not used."""
        used = set()
        for name, shape, put, _ in self.named_weights():
            t = sd.get(name)
            if t is None:
                if strict:
                    raise KeyError(f"missing weight {name}")
                continue
            if tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {tuple(shape)}")
            put(t)
            used.add(name)
        return [k for k in sd if k not in used]

    def hf_state_dict(self, merged: bool = False) -> Dict[str, torch.Tensor]:
        """Checkpoint names -> tensors, in bf16 as the design's files store them."""
        return {name: get().detach().to(torch.bfloat16).contiguous() for name, _, _, get in self.named_weights()}

    @torch.no_grad()
    def init_weights(self, std: float = 0.02, seed: int = 0, device=None) -> "HybridDecoderLM":
        """Random model: N(0, std) matrices, unit norms, decays, step sizes and sinks spread over their usual ranges. Drawn on
        ``device`` (CPU unless given: the values then do not depend on the model's device)."""
        g = torch.Generator(device=device or "cpu").manual_seed(seed)
        for name, shape, put, _ in self.named_weights():
            leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
            rnd = lambda: torch.empty(shape, device=device or "cpu")      # noqa: E731
            if leaf.endswith("mlp.router"):
                put(rnd().normal_(0.0, 1.0, generator=g).div_(shape[1] ** 0.5))      # logits of order one: spread over the experts
            elif leaf.endswith("mlp.correction"):
                put(rnd().normal_(0.0, 0.01, generator=g))
            elif leaf.endswith("mix.sink"):
                put(rnd().normal_(0.0, 1.0, generator=g))
            elif leaf.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
                put(rnd().normal_(0.0, 0.1, generator=g))
            elif leaf.endswith(".lower"):
                put(rnd().uniform_(0.0, 0.9, generator=g))
            elif leaf.endswith("mix.f.b") or leaf.endswith("right.f.b"):
                put(rnd().uniform_(1.0, 6.0, generator=g))
            elif leaf.endswith(".pb"):
                put(torch.full(shape, -4.0, device=device or "cpu"))
            elif self.cfg.design.norm_base and leaf in ("norm1", "norm2", "norm1b", "norm2b", "final.norm"):
                put(torch.full(shape, 1.0 - self.cfg.design.norm_base, device=device or "cpu"))
            elif leaf.endswith(".A_log"):
                put(rnd().uniform_(1.0, 16.0, generator=g).log_())
            elif leaf.endswith(".dt_bias"):
                put(rnd().uniform_(-4.6, -2.3, generator=g))
            elif leaf.endswith(".D") or leaf.endswith("norm") or leaf in ("norm1", "norm2"):
                put(torch.ones(shape, device=device or "cpu"))
            elif leaf.endswith(".conv") or leaf == "canon1":
                put(rnd().uniform_(-0.5, 0.5, generator=g))
            elif leaf.endswith(".b"):
                put(torch.zeros(shape, device=device or "cpu"))
            else:
                put(rnd().normal_(0.0, std, generator=g))
        return self

    def head_weight(self) -> torch.Tensor:
        return self.head

    def num_parameters(self, trainable_only: bool = False) -> int:
        return 0 if trainable_only else sum(p.numel() for p in self.parameters())

    # ------------------------------------------------------------------ cache / forward
    def new_cache(self, num_blocks: int, dtype=None, device=None, max_seqs: int = 64, quant=None, window: int = 0,
                  sink: int = 0) -> StateCache:
        if quant or window:
            raise ValueError("the latent / state cache has no quantised or windowed variant")
        p = self.embed_tokens
        if self.cfg.design.block == "sandwich":
            specs = [self.layers[i].cache_spec() for i, _ in self.runs]
            specs.append(CacheSpec(slots={"token": ((1,), torch.int32)}))      # behind the layer runs: the sequences' latest tokens
        else:
            specs = [self.layers[i].mixer.cache_spec() for i, _ in self.runs]
        return StateCache(specs, num_blocks, max_seqs, dtype or p.dtype, device or p.device, max_length=self.cfg.max_positions)

    @torch.no_grad()
    def forward_hidden(self, input_ids: torch.Tensor, positions=None, cu_seqlens: Optional[torch.Tensor] = None,
                       seq_start=None) -> torch.Tensor:
        """Final-normed hidden state of every token of whole documents, [T] (cut at ``cu_seqlens``) or [B, L], on a cache of
        their own; positions count from 0 in each document, as the model has it."""
        if input_ids.dim() == 2:
            lens = [input_ids.shape[1]] * input_ids.shape[0]
        else:
            lens = cu_seqlens.diff().tolist() if cu_seqlens is not None else [input_ids.shape[0]]
        lens = [n for n in lens if n > 0]
        cache = self.new_cache(sum(-(-n // BLOCK) for n in lens), max_seqs=len(lens))
        for i in range(len(lens)):
            cache.add_sequence(i)
        return self.forward_paged(input_ids.reshape(-1), cache, cache.prepare(list(range(len(lens))), lens), all_logits=True,
                                  return_hidden=True)

    def forward(self, input_ids: torch.Tensor, positions=None, cu_seqlens=None, seq_start=None) -> torch.Tensor:
        """Logits of every token, shaped like ``input_ids``."""
        h = self.forward_hidden(input_ids, positions, cu_seqlens, seq_start)
        return ops.project_f32(h, self.head, self.cfg.vocab_size).view(*input_ids.shape, -1)

    @torch.no_grad()
    def forward_paged(self, input_ids: torch.Tensor, cache: StateCache, meta, all_logits: bool = False,
                      return_hidden: bool = False, rows: Optional[torch.Tensor] = None, on_layer=None) -> torch.Tensor:
        """Logits (fp32) of the last new token of every sequence, of every new token (``all_logits``) or of the token rows
        listed in ``rows`` (int64). ``on_layer(i, stream)`` sees the fp32 stream after the i-th layer run."""
        from ..ops import native as nat
        if not self.embed_tokens.is_cuda or not nat.available():
            raise RuntimeError("the hybrid decoder runs on a CUDA device with the native kernel library "
                               f"({nat.load_error() or 'no CUDA device'})")
        cfg = self.cfg
        ctx = StepContext(meta, self._freqs)
        if rows is None and not all_logits:
            rows = (meta.q_start + meta.q_lens - 1).long()
        if cfg.design.block == "sandwich":
            h = self._sandwich(input_ids, cache, ctx, rows, on_layer)
        else:
            xf, xc = nat.embed_scale(input_ids, self.embed_tokens, cfg.embed_scale)
            h = (self._parallel if cfg.design.block == "parallel" else self._serial)(xf, xc, cache, ctx, rows, on_layer)
        if h.shape[0] == 0:
            return torch.empty(0, h.shape[1] if return_hidden else cfg.vocab_size, dtype=torch.float32, device=h.device)
        return h if return_hidden else ops.project_f32(h, self.head, cfg.vocab_size)

    def _serial(self, xf, xc, cache, ctx, rows, on_layer) -> torch.Tensor:
        from ..ops import native as nat
        for i, layer in enumerate(self.layers):
            xf, xc = layer(xf, xc, cache, ctx)
            if on_layer is not None:
                on_layer(i, xf)
        if rows is not None and rows.shape[0] == 0:
            return xc[:0]
        if self.norm_b is None:
            return nat.add_rmsnorm(xf, self.norm_w, self.cfg.norm_eps, rows=rows, want_stream=False, dtype=self.dtype,
                                   w_base=self.cfg.design.norm_base)[1]
        return nat.post_layernorm(xf, None, self.norm_w, self.norm_b, self.cfg.norm_eps, rows=rows, want_stream=False,
                                  dtype=self.dtype)[1]

    def _parallel(self, x0, _, cache, ctx, rows, on_layer) -> torch.Tensor:
        from ..ops import native as nat
        eps, dt = self.cfg.norm_eps, self.dtype
        x = x0
        _, h = nat.add_rmsnorm(x, self.layers[self.runs[0][0]].norm1_w, eps, dtype=dt, want_stream=False)
        for n, (i, _) in enumerate(self.runs):
            y, z, inv, k = self.layers[i](h, cache, ctx, n)
            terms = dict(y=y, z=z, inv=inv, k=k)
            last = n + 1 == len(self.runs)
            if on_layer is not None:                       # the stream between the sum and what precedes the next layer
                x, _ = nat.add_rmsnorm(x, self.norm_w, eps, dtype=dt, **terms)
                on_layer(n, x)
                terms = {}
            if last:
                if rows is not None and rows.shape[0] == 0:
                    return h[:0]
                return nat.add_rmsnorm(x, self.norm_w, eps, rows=rows, dtype=dt, want_stream=False, **terms)[1]
            nxt, again = self.runs[n + 1]
            x, h = nat.add_rmsnorm(x, self.layers[nxt].norm1_w, eps, x0=x0 if again else None, dtype=dt,
                                   out=None if x is x0 or on_layer is not None else x, **terms)

    def _sandwich(self, ids, cache, ctx, rows, on_layer) -> torch.Tensor:
        from ..ops import native as nat
        cfg, dt, meta = self.cfg, self.dtype, ctx.meta
        W, kw = cfg.hidden_size, {"base": cfg.design.norm_base, "dtype": self.dtype}
        # [stream | embedding output] in the compute type, as the projection at the start of a pass reads it
        cat = torch.empty(ids.shape[0], 2 * W, dtype=dt, device=ids.device) if self.loop_in is not None else None
        x = nat.pair_embed(ids, self.embed_tokens, self.bigram, self.pos, meta, cache.slots[len(self.runs)]["token"], cfg.pair,
                           cat[:, W:] if cat is not None else None)
        single = meta.max_q == 1

        def enter(n, x, **last):
            """(stream, input of layer run n's mixer) behind the sublayer result in ``last``."""
            i, starts = self.runs[n]
            layer, ring = self.layers[i], cache.slots[n]["canon"]
            if starts:
                x, _ = nat.branch_norm(x, cfg.norm_eps, oc=cat[:, :W], out=x, **last, **kw)
                if on_layer is not None and n:
                    on_layer(n - 1, x.clone())
                x, last = ops.project_f32(cat, self.loop_in, W).contiguous(), {}
            conv = (layer.conv_w, ring, meta.state_slots, meta.positions) if single else None
            x, h = nat.branch_norm(x, cfg.norm_eps, wn=layer.norm1_w, conv=conv, out=x, **last, **kw)
            if on_layer is not None and n and not starts:
                on_layer(n - 1, x.clone())
            return x, (h if single else nat.canon(h, layer.conv_w, ring, meta))

        x, h = enter(0, x)
        for n, (i, _) in enumerate(self.runs):
            x, last = self.layers[i](x, h, cache, ctx, n)
            if n + 1 < len(self.runs):
                x, h = enter(n + 1, x, **last)
        if on_layer is not None:
            on_layer(len(self.runs) - 1, nat.branch_norm(x, cfg.norm_eps, **last, **kw)[0])
        if rows is not None and rows.shape[0] == 0:
            return h[:0]
        return nat.branch_norm(x, cfg.norm_eps, wn=self.norm_w, rows=rows, want_stream=False, **last, **kw)[1]
