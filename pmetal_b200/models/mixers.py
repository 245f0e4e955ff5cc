"""Token mixers of the config-driven serving decoder (``hybrid_decoder.py``).

A mixer is built from its entry in the configuration, says what it keeps in the cache (``cache_spec``), lists its weights
(``named_weights``) and runs on the new tokens of a step: ``forward(x, cache, ctx, run)`` with x [tokens, width] in the
compute type returns [tokens, >= width]. ``run`` counts layer runs of the step (the layer's index in stacks without loops) and
names what the mixer keeps in the cache for this run. ``MIXERS`` names the classes; a design (``hybrid_decoder.DESIGNS``) says
which of them the ``type`` entries of its configuration mean. A new kind of mixer is one more entry.

``Mamba2Mixer``          selective state space with one decay per head (csrc/ssm.cu)
``LatentAttentionMixer`` multi-head latent attention on cached latents, its own or an earlier layer's; queries from the input
                         or from a latent of their own (csrc/latent_attn.cu)
``LinearAttentionMixer`` linear attention with a fixed decay per head; ``LightningMixer`` and ``RetentionMixer`` set its
                         activation, rotation, norm and gate (csrc/linear_attn.cu)
``GroupedAttentionMixer`` grouped-query attention of any key and value size (csrc/window_attn.cu): ``WindowAttentionMixer``
                         (sliding window, keys as values), ``DifferenceAttentionMixer`` (difference of two maps),
                         ``SinkAttentionMixer`` (capped scores, a sink per head) and ``SigmoidAttentionMixer`` (chunks, sigmoid weights)
``ChannelGateMixer``     linear attention with a forget gate per channel that also says what is written (csrc/gated_linear.cu)
``MatrixMemoryMixer``    matrix memory with exponential input gates and a normaliser (csrc/gated_linear.cu)
``ParallelMixer``        two mixers on one input: one input and one output projection around both
"""
from __future__ import annotations

import math
from typing import Callable, Dict, Optional, Tuple

import torch
import torch.nn as nn

from ..ops import functional as ops
from .state_cache import CacheSpec, attention_runs, split_groups

# portions up to this many tokens take the decode kernels (state-space scan, attention in the latent space)
SHORT = 16


def pad_rows(w: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    """Zero rows behind a weight so that products can be stored in 16-byte pieces."""
    n = -w.shape[0] % multiple
    return torch.cat([w, w.new_zeros(n, w.shape[1])]) if n else w


def frozen(t: torch.Tensor) -> nn.Parameter:
    return nn.Parameter(t.contiguous(), requires_grad=False)


class StepContext:
    """What the layers of one forward share: batch metadata, rotation tables, the split into short and long portions."""

    def __init__(self, meta, freqs: "RotationFreqs"):
        self.meta, self.freqs = meta, freqs
        self._rope: Dict[tuple, tuple] = {}
        self._groups: Dict[int, tuple] = {}
        self._runs: Dict[tuple, list] = {}

    def rope(self, base: float, dims: int):
        key = (base, dims)
        if key not in self._rope:
            from ..ops import native as nat
            self._rope[key] = nat.rope_table_f64(self.meta.positions, self.freqs.get(base, dims, self.meta.positions.device))
        return self._rope[key]

    def groups(self, limit: int):
        if limit not in self._groups:
            self._groups[limit] = split_groups(self.meta, limit)
        return self._groups[limit]

    def runs(self, limit: int, chunk: int = 0):
        """The sequences with more than ``limit`` new tokens as launches of the flash-attention kernel; ``chunk`` > 0: tokens see their
        own chunk of that many positions."""
        key = (limit, chunk)
        if key not in self._runs:
            self._runs[key] = attention_runs(self.meta, self.groups(limit)[1], chunk)
        return self._runs[key]


class RotationFreqs:
    """base^(-2 i / dims) in fp64, one device tensor per (base, dims)."""

    def __init__(self):
        self._t: Dict[tuple, torch.Tensor] = {}

    def get(self, base: float, dims: int, device) -> torch.Tensor:
        key = (base, dims, str(device))
        if key not in self._t:
            i = torch.arange(0, dims, 2, dtype=torch.float64)
            self._t[key] = torch.pow(torch.tensor(float(base), dtype=torch.float64), -i / dims).to(device)
        return self._t[key]


class Mamba2Mixer(nn.Module):
    """[z | x | B | C | dt] projection, causal convolution + silu on (x, B, C), recurrence, gate before a norm in
    ``norm_groups`` equal parts, output projection."""

    KEYS = ("heads", "vdim", "state", "groups", "conv", "norm_groups")

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        if m["heads"] % m["groups"]:
            raise ValueError(f"layer {index}: {m['heads']} heads do not divide into {m['groups']} groups")
        if m["heads"] * m["vdim"] % m["norm_groups"]:
            raise ValueError(f"layer {index}: inner width does not divide into {m['norm_groups']} norm parts")

    def __init__(self, m: dict, cfg, index: int, dtype, device):
        super().__init__()
        self.dims = (m["heads"], m["vdim"], m["state"], m["groups"], m["conv"])
        self.H, self.P, self.N, self.G, self.taps = self.dims
        self.parts, self.eps, self.index = m["norm_groups"], cfg.norm_eps, index
        self.inner = self.H * self.P
        self.conv_dim = self.inner + 2 * self.G * self.N
        self.width, self.dtype = cfg.hidden_size, dtype
        kw = dict(device=device)
        n_in = self.inner + self.conv_dim + self.H
        self.w_in = frozen(torch.zeros(-(-n_in // 8) * 8, self.width, dtype=dtype, **kw))
        self.conv_w = frozen(torch.zeros(self.taps, self.conv_dim, **kw))          # [taps][channel]
        self.conv_b = frozen(torch.zeros(self.conv_dim, **kw))
        self.dt_bias, self.a_log, self.dskip = (frozen(torch.zeros(self.H, **kw)) for _ in range(3))
        self.norm_w = frozen(torch.zeros(self.inner, **kw))
        self.w_o = frozen(torch.zeros(-(-self.width // 8) * 8, self.inner, dtype=dtype, **kw))

    def cache_spec(self) -> CacheSpec:
        p4 = -(-self.P // 4) * 4
        return CacheSpec(slots={"conv": ((self.taps, self.conv_dim), None), "state": ((self.H, self.N, p4), torch.float32)})

    def named_weights(self):
        """(checkpoint suffix, shape, setter, getter)."""
        n_in = self.inner + self.conv_dim + self.H
        yield "in", (n_in, self.width), lambda t: self.w_in[:n_in].copy_(t), lambda: self.w_in[:n_in]
        yield "conv", (self.conv_dim, self.taps), lambda t: self.conv_w.copy_(t.t()), lambda: self.conv_w.t()
        yield "conv.b", (self.conv_dim,), self.conv_b.copy_, lambda: self.conv_b
        yield "dt_bias", (self.H,), self.dt_bias.copy_, lambda: self.dt_bias
        yield "A_log", (self.H,), self.a_log.copy_, lambda: self.a_log
        yield "D", (self.H,), self.dskip.copy_, lambda: self.dskip
        yield "norm", (self.inner,), self.norm_w.copy_, lambda: self.norm_w
        yield "o", (self.width, self.inner), lambda t: self.w_o[:self.width].copy_(t), lambda: self.w_o[:self.width]

    def forward(self, x: torch.Tensor, cache, ctx: StepContext, run: Optional[int] = None) -> torch.Tensor:
        from ..ops import native as nat
        store = cache.slots[self.index if run is None else run]
        u = ops.project(x, self.w_in)
        y = torch.empty(x.shape[0], self.inner, dtype=x.dtype, device=x.device)
        args = (u, self.conv_w, self.conv_b, self.dt_bias, self.a_log, self.dskip, store["conv"], store["state"])
        tensor_cores = x.dtype == torch.bfloat16 and nat.ssm_chunk_supported(self.N)
        short, long = ctx.groups(SHORT if tensor_cores else 1 << 30)
        if short is not None:
            nat.ssm_scan(*args, short, self.dims, y)
        if long is not None:
            nat.ssm_chunk(*args, long, self.dims, y)
        g = nat.ssm_gate_norm(y, u, self.norm_w, self.eps, self.parts, store["conv"], ctx.meta, self.dims)
        return ops.project(g, self.w_o)


class LatentAttentionMixer(nn.Module):
    """Causal attention whose cache is one latent and one rotated key part per token. ``kv_from`` makes the layer read an
    earlier layer's rows with its own up-projections. ``q_rank``: the queries come from a normed latent of that size."""

    KEYS = ("heads", "dim", "rot_dim", "vdim", "kv_rank", "rot", "scale")

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        if m["rot_dim"] % 2:
            raise ValueError(f"layer {index}: rot_dim must be even")
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"layer {index}: rot.dims must equal rot_dim")
        if m.get("q_rank") is not None and m["q_rank"] < 1:
            raise ValueError(f"layer {index}: q_rank must be at least 1")
        src = m.get("kv_from")
        if src is None:
            return
        if not 0 <= src < index or layers[src]["type"] != "latent_attention" or layers[src]["mixer"].get("kv_from") is not None:
            raise ValueError(f"layer {index}: kv_from must name an earlier latent attention layer with its own latents")
        o = layers[src]["mixer"]
        if any(o[k] != m[k] for k in ("kv_rank", "rot_dim", "rot")):
            raise ValueError(f"layer {index}: kv_rank, rot_dim and rotation must equal layer {src}'s")

    def __init__(self, m: dict, cfg, index: int, dtype, device):
        super().__init__()
        H, dn, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        self.row = -(-(r + dr) // 16) * 16
        self.dims = (H, dn, dr, dv, r, self.row)
        self.base, self.scale, self.eps = float(m["rot"]["base"]), float(m["scale"]), cfg.norm_eps
        src = m.get("kv_from")
        self.own, self.source, self.index = src is None, index if src is None else src, index
        self.width = cfg.hidden_size
        self.n_q, self.n_d, self.n_k, self.n_v = H * (dn + dr), (r + dr) if src is None else 0, H * dn, H * dv
        kw = dict(dtype=dtype, device=device)
        up8 = lambda n: -(-n // 8) * 8      # noqa: E731
        self.q_rank = m.get("q_rank") or 0
        self.n_in = self.q_rank or self.n_q
        self.w_q = frozen(torch.zeros(up8(self.n_in + self.n_d), self.width, **kw))      # queries (or their latent), then the down-projection
        self.w_uq = frozen(torch.zeros(up8(self.n_q), self.q_rank, **kw)) if self.q_rank else None
        self.q_norm_w = frozen(torch.zeros(self.q_rank, device=device)) if self.q_rank else None
        self.w_ukv = frozen(torch.zeros(up8(self.n_k + self.n_v), r, **kw))              # keys of all heads, then values
        self.w_o = frozen(torch.zeros(up8(self.width), self.n_v, **kw))
        self.norm_w = frozen(torch.zeros(r, device=device)) if self.own else None
        self._ukv8: Optional[torch.Tensor] = None
        self.expand = dtype == torch.bfloat16 and dn + dr <= 128 and dv <= 128

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(page_width=self.row + 8 if self.own else 0)      # the kernels keep rows eight columns apart

    def named_weights(self):
        q, d, k, v, n_q = self.n_in, self.n_d, self.n_k, self.n_v, self.n_q
        r = self.dims[4]
        yield "dq" if self.q_rank else "q", (q, self.width), lambda t: self.w_q[:q].copy_(t), lambda: self.w_q[:q]
        if self.q_rank:
            yield "dq.norm", (q,), self.q_norm_w.copy_, lambda: self.q_norm_w
            yield "uq", (n_q, q), lambda t: self.w_uq[:n_q].copy_(t), lambda: self.w_uq[:n_q]
        if self.own:
            yield "dkv", (d, self.width), lambda t: self.w_q[q:q + d].copy_(t), lambda: self.w_q[q:q + d]
            yield "dkv.norm", (r,), self.norm_w.copy_, lambda: self.norm_w
        yield "uk", (k, r), lambda t: self.w_ukv[:k].copy_(t), lambda: self.w_ukv[:k]
        yield "uv", (v, r), lambda t: self.w_ukv[k:k + v].copy_(t), lambda: self.w_ukv[k:k + v]
        yield "o", (self.width, v), lambda t: self.w_o[:self.width].copy_(t), lambda: self.w_o[:self.width]

    def _expand_weight(self) -> torch.Tensor:
        """[keys; values] up-projection with its rank padded to 16-byte rows (the weight itself when it is already)."""
        r = self.dims[4]
        if r % 8 == 0:
            return self.w_ukv
        if self._ukv8 is None or self._ukv8.device != self.w_ukv.device:
            self._ukv8 = torch.nn.functional.pad(self.w_ukv, (0, -r % 8)).contiguous()
        return self._ukv8

    def forward(self, x: torch.Tensor, cache, ctx: StepContext, run: Optional[int] = None) -> torch.Tensor:
        from ..ops import native as nat
        H, dn, dr, dv, r, W = self.dims
        pages = cache.pages[run if self.own and run is not None else self.source]
        qd = ops.project(x, self.w_q)
        rope = ctx.rope(self.base, dr) if dr else (None, None)
        nat.latent_prep(qd, self.norm_w, self.eps, *rope, self.dims, pages if self.own else None, ctx.meta.slots, self.q_rank,
                        self.q_norm_w)
        o = torch.empty(x.shape[0], H * dv, dtype=x.dtype, device=x.device)
        short, long = ctx.groups(SHORT if self.expand else 1 << 30)
        turn = (None, None)
        if self.q_rank:
            qd = ops.project(qd[:, :self.q_rank], self.w_uq)
            if long is None:
                turn = rope                                # on the way into the short portions' kernel
            elif dr:
                nat.latent_prep(qd, None, self.eps, *rope, self.dims, None, ctx.meta.slots)
        if short is not None:
            nat.latent_attn(qd, self.w_ukv, self.w_ukv[self.n_k:], pages, short, self.dims, self.scale, o, turn)
        if long is not None:
            w = self._expand_weight()
            for r in ctx.runs(SHORT):
                nat.latent_expand_attn(qd, w, pages, r, self.dims, self.scale, o)
        return ops.project(o, self.w_o)


def check_rotation(m: dict, index: int) -> None:
    if m["rot"]["dims"] % 2 or not 0 <= m["rot"]["dims"] <= m["dim"]:
        raise ValueError(f"layer {index}: rot.dims must be even and at most dim")


class LinearAttentionMixer(nn.Module):
    """S <- decay S + k v^T, o = S^T q per head; the heads are RMS-normed (together or one by one), gated and projected."""

    KEYS = ("heads", "dim", "vdim", "decay")
    SILU = False               # activation of q, k and v
    ROTATION = "none"          # layout of the rotated pairs of q and k
    KEY_FACTOR = False         # k times dim^(-1/2)
    HEAD_NORM = False          # every head by itself and without a weight, else all heads together with a weight
    SILU_GATE = False          # silu gate, else sigmoid

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        if len(m["decay"]) != m["heads"]:
            raise ValueError(f"layer {index}: {len(m['decay'])} decays for {m['heads']} heads")
        if not all(0.0 <= float(d) <= 1.0 for d in m["decay"]):
            raise ValueError(f"layer {index}: decays must lie in [0, 1]")
        if cls.ROTATION != "none":
            check_rotation(m, index)

    def __init__(self, m: dict, cfg, index: int, dtype, device):
        super().__init__()
        self.H, self.N, self.P = m["heads"], m["dim"], m["vdim"]
        rot = m["rot"] if self.ROTATION != "none" else {"base": 1.0, "dims": 0}
        self.base, self.R = float(rot["base"]), int(rot["dims"])
        self.dims = (self.H, self.N, self.P, self.R, self.ROTATION if self.R else "none", self.SILU)
        self.kscale = self.N ** -0.5 if self.KEY_FACTOR else 1.0
        self.eps, self.index, self.width = cfg.norm_eps, index, cfg.hidden_size
        self.inner, self.n_k = self.H * self.P, self.H * self.N
        n_in = 2 * self.n_k + 2 * self.inner
        kw = dict(device=device)
        self.w_in = frozen(torch.zeros(-(-n_in // 8) * 8, self.width, dtype=dtype, **kw))      # q, k, v, gate
        self.w_o = frozen(torch.zeros(-(-self.width // 8) * 8, self.inner, dtype=dtype, **kw))
        self.norm_w = None if self.HEAD_NORM else frozen(torch.zeros(self.inner, **kw))
        self.decay = frozen(torch.tensor([float(d) for d in m["decay"]], dtype=torch.float64).float().to(device or "cpu"))
        # a decay below 2^-100 leaves nothing that fp32 sums would show
        self.log2_decay = frozen(torch.tensor([max(math.log2(d), -100.0) if d > 0 else -100.0 for d in m["decay"]],
                                              dtype=torch.float64).float().to(device or "cpu"))

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(slots={"state": ((self.H, self.N, -(-self.P // 4) * 4), torch.float32)})

    def named_weights(self):
        at = 0
        for name, n in (("q", self.n_k), ("k", self.n_k), ("v", self.inner), ("g", self.inner)):
            yield (name, (n, self.width), lambda t, a=at, n=n: self.w_in[a:a + n].copy_(t), lambda a=at, n=n: self.w_in[a:a + n])
            at += n
        if self.norm_w is not None:
            yield "norm", (self.inner,), self.norm_w.copy_, lambda: self.norm_w
        yield "o", (self.width, self.inner), lambda t: self.w_o[:self.width].copy_(t), lambda: self.w_o[:self.width]

    def forward(self, x: torch.Tensor, cache, ctx: StepContext, run: Optional[int] = None) -> torch.Tensor:
        from ..ops import native as nat
        state = cache.slots[self.index if run is None else run]["state"]
        u = ops.project(x, self.w_in)
        cos, sin = ctx.rope(self.base, self.R) if self.R else (None, None)
        y = torch.empty(x.shape[0], self.inner, dtype=x.dtype, device=x.device)
        tensor_cores = x.dtype == torch.bfloat16 and nat.linear_chunk_supported(self.N)
        short, long = ctx.groups(SHORT if tensor_cores else 1 << 30)
        if short is not None:
            nat.linear_scan(u, cos, sin, self.decay, self.kscale, state, short, self.dims, y)
        if long is not None:
            nat.linear_chunk(u, cos, sin, self.log2_decay, self.kscale, state, long, self.dims, y)
        gate = u[:, 2 * self.n_k + self.inner:]
        g = nat.norm_gate(y, gate, self.norm_w, self.eps, self.H if self.HEAD_NORM else 1, self.SILU_GATE)
        return ops.project(g, self.w_o)


class LightningMixer(LinearAttentionMixer):
    SILU = True


class RetentionMixer(LinearAttentionMixer):
    KEYS = LinearAttentionMixer.KEYS + ("rot",)
    ROTATION = "half"
    KEY_FACTOR = HEAD_NORM = SILU_GATE = True


Place = Callable[[], Tuple[torch.Tensor, torch.Tensor]]


class StackedMixer(nn.Module):
    """A mixer between one stacked input projection and one output projection, which may be parts of larger ones: ``place`` gives
    the rows and columns that are this mixer's (``ParallelMixer``), else it owns both. ``n_in`` rows enter as activations (padded to 8),
    ``n_gate`` further ones as fp32 logits; ``inner`` columns leave."""

    n_in = n_gate = inner = 0

    def _own_projections(self, width: int, dtype, device, place: Optional[Place]) -> None:
        up8 = lambda n: -(-n // 8) * 8      # noqa: E731
        self.width, self.n_pad = width, up8(self.n_in)
        self.place = place
        if place is None:
            self.w_in = frozen(torch.zeros(up8(self.n_pad + self.n_gate) if self.n_gate else self.n_pad, width, dtype=dtype, device=device))
            self.w_o = frozen(torch.zeros(up8(width), self.inner, dtype=dtype, device=device))

    def _rows(self, at: int, n: int):
        """(setter, getter) of ``n`` rows of the input projection."""
        part = lambda: (self.place()[0] if self.place else self.w_in)[at:at + n]      # noqa: E731
        return (lambda t: part().copy_(t)), part

    def _output(self):
        part = lambda: (self.place()[1] if self.place else self.w_o)[:self.width, :self.inner]      # noqa: E731
        return "o", (self.width, self.inner), (lambda t: part().copy_(t)), part


class GroupedAttentionMixer(StackedMixer):
    """Grouped-query attention on cached keys and values. The class says what the design fixes, the configuration entry
    gives sizes and, where present, the rotation (``rot``), the window or the size of the chunks (``mask``), the query factor that grows
    with the position (``q_temp``) and the cap of the scores (``softcap``). ``kv_from`` makes the layer read an earlier layer's keys and
    values with its own queries."""

    KEYS = ("heads", "kv_heads", "dim", "vdim", "scale")
    MAPS = 1                   # attention maps per head over the same values; with two their difference is taken
    ROTATION = "none"          # layout of the rotated pairs of q and k
    UNIT_NORM = True           # queries and keys divided by their root mean square over the head
    NORM_WEIGHTS = True        # and multiplied with a weight
    OWN_VALUES = True          # else the values are the keys as projected
    SINK = False               # a learned score per head without a value
    GATE = True                # sigmoid of a projection of the input, one number per head
    CHUNKED = False            # a position sees its own chunk of ``mask.size`` positions, else a window of that size
    SIGMOID = False            # sigmoid of score + a number per head in place of the softmax

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {index}: {m['heads']} heads do not divide into {m['kv_heads']} key/value heads")
        if not cls.OWN_VALUES and m["vdim"] != m["dim"]:
            raise ValueError(f"layer {index}: vdim must equal dim where the values are the keys")
        if max(m["dim"], m["vdim"]) > 1024:
            raise ValueError(f"layer {index}: heads of more than 1024 channels")
        if cls.ROTATION != "none":
            check_rotation(m, index)
        if m.get("mask") is not None and m["mask"].get("size", 0) < 1:
            raise ValueError(f"layer {index}: mask.size must be at least 1")
        temp = m.get("q_temp")
        if temp is not None and (temp["every"] < 1 or temp["every"] != int(temp["every"])):
            raise ValueError(f"layer {index}: q_temp.every must be a positive whole number")
        if m.get("softcap") is not None and not m["softcap"] > 0:
            raise ValueError(f"layer {index}: softcap must be positive")
        src = m.get("kv_from")
        if src is None:
            return
        if not 0 <= src < index or layers[src]["type"] != layers[index]["type"] or layers[src]["mixer"].get("kv_from") is not None:
            raise ValueError(f"layer {index}: kv_from must name an earlier layer of the same kind with its own keys and values")
        o = layers[src]["mixer"]
        if any(o.get(k) != m.get(k) for k in ("heads", "kv_heads", "dim", "vdim", "rot", "mask")):
            raise ValueError(f"layer {index}: head counts, sizes, rotation and window must equal layer {src}'s")

    def __init__(self, m: dict, cfg, index: int, dtype, device, place: Optional[Place] = None):
        super().__init__()
        H, G, M, D, DV = self.dims = (m["heads"], m["kv_heads"], self.MAPS, m["dim"], m["vdim"])
        rot = m["rot"] if self.ROTATION != "none" else {"base": 1.0, "dims": 0}
        self.base, self.R = float(rot["base"]), int(rot["dims"])
        self.scale, self.eps = float(m["scale"]), cfg.norm_eps
        self.window = int(m["mask"]["size"]) if m.get("mask") is not None else 0
        self.softcap = float(m["softcap"]) if m.get("softcap") is not None else 0.0
        temp = m.get("q_temp")
        self.temp = (float(temp["coef"]), int(temp["every"])) if temp is not None else None
        src = m.get("kv_from")
        self.own, self.source, self.index = src is None, index if src is None else src, index
        parts = [("q", H * M * D)]
        if self.own:
            parts += [("k", G * M * D)] + ([("v", G * DV)] if self.OWN_VALUES else [])
        if self.GATE:
            parts.append(("g", H))
        self.parts, self.at, n = parts, {}, 0
        for name, rows in parts:
            self.at[name] = n
            n += rows
        self.n_in, self.inner = n, H * DV
        self._own_projections(cfg.hidden_size, dtype, device, place)
        vec = lambda n: frozen(torch.zeros(n, device=device))      # noqa: E731
        self.wbias = vec(H) if self.SIGMOID else None
        self.q_norm_w = vec(D) if self.NORM_WEIGHTS else None
        self.k_norm_w = vec(D) if self.NORM_WEIGHTS and self.own else None
        self.sink = vec(H) if self.SINK else None
        self.diff = float(m["diff"]) if M > 1 else 0.0
        if M > 1:
            self.lq1, self.lk1, self.lq2, self.lk2 = (vec(D) for _ in range(4))
            self.register_buffer("lam", torch.zeros(1, device=device), persistent=False)

    def cache_spec(self) -> CacheSpec:
        _, G, M, D, DV = self.dims
        pad8 = lambda n: -(-n // 8) * 8      # noqa: E731
        return CacheSpec(page_width=G * (M * pad8(D) + pad8(DV)), window=self.window) if self.own else CacheSpec()

    @torch.no_grad()
    def _put_lambda(self, dst: torch.Tensor, t: torch.Tensor) -> None:
        dst.copy_(t)
        self.lam.copy_((torch.exp((self.lq1 * self.lk1).sum()) - torch.exp((self.lq2 * self.lk2).sum()) + self.diff).view(1))

    def named_weights(self):
        for name, n in self.parts:
            yield (name, (n, self.width), *self._rows(self.at[name], n))
        for name in ("q", "k"):
            p = getattr(self, name + "_norm_w")
            if p is not None:
                yield name + ".norm", tuple(p.shape), p.copy_, lambda p=p: p
        if self.sink is not None:
            yield "sink", tuple(self.sink.shape), self.sink.copy_, lambda: self.sink
        if self.wbias is not None:
            yield "pb", tuple(self.wbias.shape), self.wbias.copy_, lambda: self.wbias
        for name in ("lq1", "lk1", "lq2", "lk2") if self.dims[2] > 1 else ():
            p = getattr(self, name)
            yield name, tuple(p.shape), lambda t, p=p: self._put_lambda(p, t), lambda p=p: p
        yield self._output()

    def forward(self, x: torch.Tensor, cache, ctx: StepContext, run: Optional[int] = None) -> torch.Tensor:
        o = torch.empty(x.shape[0], self.inner, dtype=x.dtype, device=x.device)
        self.mix(ops.project(x, self.w_in), None, cache, ctx, run, o)
        return ops.project(o, self.w_o)

    def mix(self, u: torch.Tensor, z, cache, ctx: StepContext, run: Optional[int], o: torch.Tensor, scale: float = 1.0) -> None:
        """Between the projections: rows u (any stride) -> ``scale`` times the heads' results in the rows of o (any stride)."""
        from ..ops import native as nat
        pages = cache.pages[run if self.own and run is not None else self.source]
        cos, sin = ctx.rope(self.base, self.R) if self.R else (None, None)
        k_at = self.at.get("k", 0)
        wide = nat.window_wide(self.dims, u.dtype, self.window, self.CHUNKED) if ctx.groups(SHORT)[1] is not None else 0
        q = nat.window_prep(u, cos, sin, self.dims, (self.R, self.ROTATION), self.UNIT_NORM, self.eps, (k_at, self.at.get("v", k_at)),
                            pages if self.own else None, ctx.meta.slots, self.q_norm_w, self.k_norm_w, self.temp, ctx.meta.positions, wide)
        self.attend(q, pages, ctx, u[:, self.at["g"]:] if self.GATE else None, o, scale)

    def attend(self, q: torch.Tensor, pages, ctx: StepContext, gate, o: torch.Tensor, scale: float) -> None:
        """Attention of prepared queries over the cached rows, short and long portions."""
        from ..ops import native as nat
        short, long = ctx.groups(SHORT)
        diff = (self.lam, 1.0 - self.diff, self.eps) if self.dims[2] > 1 else None
        more = (self.softcap, self.sink, gate, diff)
        if short is not None:
            nat.window_attn(q, pages, short, self.dims, self.window, self.scale, True, o, *more, self.CHUNKED, self.wbias, scale)
        if long is not None and nat.window_wide(self.dims, q.dtype, self.window, self.CHUNKED):
            runs = ctx.runs(SHORT, self.window if self.CHUNKED else 0)
            nat.window_expand_attn(q, pages, long, runs, self.dims, self.scale, o, *more, self.wbias, scale)
        elif long is not None:
            nat.window_attn(q, pages, long, self.dims, self.window, self.scale, False, o, *more, self.CHUNKED, self.wbias, scale)


class WindowAttentionMixer(GroupedAttentionMixer):
    """Sliding window. Queries and keys are rotated, then divided by their root mean square; the values are the keys as
    projected."""

    KEYS = GroupedAttentionMixer.KEYS + ("rot", "mask")
    ROTATION = "pairs"
    NORM_WEIGHTS = OWN_VALUES = GATE = False


class DifferenceAttentionMixer(GroupedAttentionMixer):
    """Two maps per head over the same values: a_1 - lambda a_2 with lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, divided by
    its root mean square over the head, times 1 - diff."""

    KEYS = GroupedAttentionMixer.KEYS + ("diff",)
    MAPS = 2


class SinkAttentionMixer(GroupedAttentionMixer):
    SINK = True


class SigmoidAttentionMixer(GroupedAttentionMixer):
    """Normed and rotated queries and keys, chunks counted from position 0, unnormalised sigmoid weights."""

    KEYS = GroupedAttentionMixer.KEYS + ("rot", "mask")
    ROTATION = "half"
    GATE = False
    CHUNKED = SIGMOID = True

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        super().check(m, index, layers)
        if m["mask"] is None:
            raise ValueError(f"layer {index}: mask.size must be at least 1")
        if any(m.get(k) is not None for k in ("kv_from", "softcap")):
            raise ValueError(f"layer {index}: attention with sigmoid weights takes neither kv_from nor softcap")


class ChannelGateMixer(StackedMixer):
    """f = lower + (1 - lower) sigmoid(W_f x + b) per head and channel, S <- diag(f) S + (1 - f) v^T, o = S^T silu(W_q x) per head; every
    head RMS-normed with one weight for all heads, and projected. Gates are formed in fp32 from fp32 sums."""

    KEYS = ("heads", "dim", "vdim")

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        if min(m["heads"], m["dim"], m["vdim"]) < 1 or m["dim"] > 2048:
            raise ValueError(f"layer {index}: heads, dim and vdim must be positive, dim at most 2048")

    def __init__(self, m: dict, cfg, index: int, dtype, device, place: Optional[Place] = None):
        super().__init__()
        self.dims = self.H, self.N, self.P = m["heads"], m["dim"], m["vdim"]
        self.n_k, self.inner = self.H * self.N, self.H * self.P
        self.v_at = -(-self.n_k // 8) * 8
        self.n_in, self.n_gate = self.v_at + self.inner, self.n_k
        self.eps, self.index = cfg.norm_eps, index
        self._own_projections(cfg.hidden_size, dtype, device, place)
        vec = lambda n: frozen(torch.zeros(n, device=device))      # noqa: E731
        self.f_bias, self.lower, self.norm_w = vec(self.n_k), vec(self.n_k), vec(self.P)

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(slots={"state": ((self.H, self.N, -(-self.P // 4) * 4), torch.float32)})

    def named_weights(self):
        for name, at, n in (("q", 0, self.n_k), ("f", self.n_pad, self.n_k), ("v", self.v_at, self.inner)):
            yield (name, (n, self.width), *self._rows(at, n))
        for name, p in (("f.b", self.f_bias), ("lower", self.lower), ("norm", self.norm_w)):
            yield name, tuple(p.shape), p.copy_, (lambda p=p: p)
        yield self._output()

    def forward(self, x: torch.Tensor, cache, ctx: StepContext, run: Optional[int] = None) -> torch.Tensor:
        o = torch.empty(x.shape[0], self.inner, dtype=x.dtype, device=x.device)
        u, z = ops.project_mixed(x, self.w_in, self.n_pad)
        self.mix(u, z, cache, ctx, run, o)
        return ops.project(o, self.w_o)

    def mix(self, u: torch.Tensor, z: torch.Tensor, cache, ctx: StepContext, run: Optional[int], o: torch.Tensor, scale: float = 1.0) -> None:
        """Between the projections: rows u and gate logits z (any stride) -> ``scale`` times the heads' results in the rows of o."""
        from ..ops import native as nat
        state = cache.slots[self.index if run is None else run]["state"]
        y = torch.empty(u.shape[0], self.inner, dtype=u.dtype, device=u.device)
        args = (u, u[:, self.v_at:], z, self.f_bias, self.lower, state)
        tensor_cores = u.dtype == torch.bfloat16 and nat.linear_chunk_supported(self.N)
        short, long = ctx.groups(SHORT if tensor_cores else 1 << 30)
        if short is not None:
            nat.channel_scan(*args, short, self.dims, y)
        if long is not None:
            nat.channel_chunk(*args, long, self.dims, y)
        nat.norm_gate(y, None, self.norm_w, self.eps, self.H, False, scale=scale, out=o)


class MatrixMemoryMixer(StackedMixer):
    """S <- exp(f + m - m') S + exp(i - m') k v^T with i = cap tanh(. / cap), f = log sigmoid(cap tanh(. / cap)) of fp32 sums and the
    running maximum m' = max(f + m, i); the read-out is divided by max(|n . q|, exp(-m')) + 1e-6, every head RMS-normed, times a weight
    and the sigmoid of a gate."""

    KEYS = ("heads", "dim", "vdim", "gate_cap")
    DEN_EPS = 1e-6

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        if min(m["heads"], m["dim"], m["vdim"]) < 1 or m["dim"] > 2048:
            raise ValueError(f"layer {index}: heads, dim and vdim must be positive, dim at most 2048")
        if not m["gate_cap"] > 0:
            raise ValueError(f"layer {index}: gate_cap must be positive")

    def __init__(self, m: dict, cfg, index: int, dtype, device, place: Optional[Place] = None):
        super().__init__()
        self.dims = self.H, self.N, self.P = m["heads"], m["dim"], m["vdim"]
        up8 = lambda n: -(-n // 8) * 8      # noqa: E731
        self.n_k, self.inner = self.H * self.N, self.H * self.P
        self.at = {"q": 0, "k": up8(self.n_k), "v": 2 * up8(self.n_k), "g": 2 * up8(self.n_k) + up8(self.inner)}
        self.n_in, self.n_gate = self.at["g"] + self.inner, 2 * self.H
        self.gates = (float(m["gate_cap"]), self.N ** -0.5, self.DEN_EPS)
        self.eps, self.index = cfg.norm_eps, index
        self._own_projections(cfg.hidden_size, dtype, device, place)
        vec = lambda n: frozen(torch.zeros(n, device=device))      # noqa: E731
        self.g_bias, self.norm_w = vec(2 * self.H), vec(self.inner)      # input gates, then forget gates

    def cache_spec(self) -> CacheSpec:
        p4 = -(-self.P // 4) * 4
        f32 = torch.float32
        return CacheSpec(slots={"state": ((self.H, self.N, p4), f32), "norm": ((self.H, self.N), f32), "max": ((self.H, p4 // 4), f32)})

    def named_weights(self):
        for name, n in (("q", self.n_k), ("k", self.n_k), ("v", self.inner), ("g", self.inner)):
            yield (name, (n, self.width), *self._rows(self.at[name], n))
        yield self._output()
        yield "norm", (self.inner,), self.norm_w.copy_, lambda: self.norm_w
        H = self.H
        for i, name in enumerate(("i", "f")):
            yield (name, (H, self.width), *self._rows(self.n_pad + i * H, H))
            yield name + ".b", (H,), lambda t, i=i: self.g_bias[i * H:(i + 1) * H].copy_(t), lambda i=i: self.g_bias[i * H:(i + 1) * H]

    def forward(self, x: torch.Tensor, cache, ctx: StepContext, run: Optional[int] = None) -> torch.Tensor:
        o = torch.empty(x.shape[0], self.inner, dtype=x.dtype, device=x.device)
        u, z = ops.project_mixed(x, self.w_in, self.n_pad)
        self.mix(u, z, cache, ctx, run, o)
        return ops.project(o, self.w_o)

    def mix(self, u: torch.Tensor, z: torch.Tensor, cache, ctx: StepContext, run: Optional[int], o: torch.Tensor, scale: float = 1.0) -> None:
        """Between the projections: rows u and gate logits z (any stride) -> ``scale`` times the heads' results in the rows of o."""
        from ..ops import native as nat
        store, at = cache.slots[self.index if run is None else run], self.at
        y = torch.empty(u.shape[0], self.inner, dtype=u.dtype, device=u.device)
        den = torch.empty(u.shape[0], self.H, dtype=torch.float32, device=u.device)
        more = (u[:, at["v"]:], z, self.g_bias, self.gates, store)
        tensor_cores = u.dtype == torch.bfloat16 and nat.linear_chunk_supported(self.N)
        short, long = ctx.groups(SHORT if tensor_cores else 1 << 30)
        if short is not None:
            nat.memory_scan(u, u[:, at["k"]:], *more, short, self.dims, y, den)
        if long is not None:
            nat.memory_chunk(u, at["q"], at["k"], *more, long, self.dims, y, den)
        nat.norm_gate(y, u[:, at["g"]:], self.norm_w, self.eps, self.H, False, den, scale, o)


class ParallelMixer(nn.Module):
    """left_scale * left(x) + right_scale * right(x). Both mixers' input projections are one product and so are the output projections:
    the scales go to the heads' results, whose columns lie side by side."""

    KEYS = ("left", "right", "left_scale", "right_scale")
    LEFT, RIGHT = SigmoidAttentionMixer, MatrixMemoryMixer

    @classmethod
    def check(cls, m: dict, index: int, layers) -> None:
        for side, kind in (("left", cls.LEFT), ("right", cls.RIGHT)):
            missing = [k for k in kind.KEYS if k not in m[side]]
            if missing:
                raise ValueError(f"layer {index}: {side} mixer entry lacks {', '.join(missing)}")
            kind.check(m[side], index, layers)

    def __init__(self, m: dict, cfg, index: int, dtype, device):
        super().__init__()
        up8 = lambda n: -(-n // 8) * 8      # noqa: E731
        self.left = self.LEFT(m["left"], cfg, index, dtype, device, lambda: (self.w_in[:self.cut], self.w_o[:, :self.c_cut]))
        self.right = self.RIGHT(m["right"], cfg, index, dtype, device, lambda: (self.w_in[self.cut:], self.w_o[:, self.c_cut:]))
        self.scales = (float(m["left_scale"]), float(m["right_scale"]))
        self.cut, self.c_cut = self.left.n_pad, up8(self.left.inner)      # the left mixer has no gate rows
        self.n_low, self.cols = self.cut + self.right.n_pad, self.c_cut + up8(self.right.inner)
        self.ragged = self.cols != self.left.inner + self.right.inner
        width = cfg.hidden_size
        self.w_in = frozen(torch.zeros(up8(self.n_low + self.right.n_gate), width, dtype=dtype, device=device))
        self.w_o = frozen(torch.zeros(up8(width), self.cols, dtype=dtype, device=device))

    def cache_spec(self) -> CacheSpec:
        a, b = self.left.cache_spec(), self.right.cache_spec()
        return CacheSpec(page_width=a.page_width, window=a.window, slots={**a.slots, **b.slots})

    def named_weights(self):
        for pre, mod in (("left.", self.left), ("right.", self.right)):
            for name, *rest in mod.named_weights():
                yield (pre + name, *rest)

    def forward(self, x: torch.Tensor, cache, ctx: StepContext, run: Optional[int] = None) -> torch.Tensor:
        u, z = ops.project_mixed(x, self.w_in, self.n_low)
        make = torch.zeros if self.ragged else torch.empty
        o = make(x.shape[0], self.cols, dtype=x.dtype, device=x.device)
        self.left.mix(u[:, :self.cut], None, cache, ctx, run, o, self.scales[0])
        self.right.mix(u[:, self.cut:], z, cache, ctx, run, o[:, self.c_cut:], self.scales[1])
        return ops.project(o, self.w_o)


MIXERS = {"mamba2": Mamba2Mixer, "latent_attention": LatentAttentionMixer, "lightning": LightningMixer,
          "retention": RetentionMixer, "window_attention": WindowAttentionMixer, "difference_attention": DifferenceAttentionMixer,
          "sink_attention": SinkAttentionMixer, "sigmoid_attention": SigmoidAttentionMixer, "channel_gate": ChannelGateMixer,
          "matrix_memory": MatrixMemoryMixer, "sigmoid_attention_and_memory": ParallelMixer}
