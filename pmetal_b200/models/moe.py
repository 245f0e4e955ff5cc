"""Mixture-of-experts feed-forward block (Qwen3-MoE).

Routing follows crates/pmetal-models/src/moe_routing.rs:36-108 and
architectures/qwen3_moe.rs:519-540: softmax over all experts in fp32, top-k, and
optional renormalisation of the k weights (``norm_topk_prob``, eps 1e-8). Experts are
stored stacked, ``gate_up`` [E, 2I, H] and ``down`` [E, H, I]; tokens are sorted by
expert and each expert's contiguous slab goes through a grouped GEMM.
"""
from __future__ import annotations

from typing import Dict, Optional, Set, Tuple

import torch
import torch.nn as nn
import torch.nn.functional as F

from .config import ModelArgs


def route_topk(router_logits: torch.Tensor, k: int, norm_topk_prob: bool = True) -> Tuple[torch.Tensor, torch.Tensor]:
    probs = torch.softmax(router_logits.float(), dim=-1)
    w, idx = torch.topk(probs, k, dim=-1)
    if norm_topk_prob:
        w = w / (w.sum(-1, keepdim=True) + 1e-8)
    return w, idx


def sort_by_expert(idx: torch.Tensor, num_experts: int):
    """Flatten [T,k] assignments; returns (order, counts, offsets) with tokens grouped by expert."""
    flat = idx.reshape(-1)
    order = torch.argsort(flat, stable=True)
    counts = torch.bincount(flat, minlength=num_experts)
    offsets = torch.zeros(num_experts + 1, dtype=torch.int64, device=idx.device)
    offsets[1:] = torch.cumsum(counts, 0)
    return order, counts, offsets


class WeightedInputExperts(nn.Module):
    """Routed experts for serving whose routing weight multiplies the expert's input: the sum over a token's experts of
    down_e(silu(G_e w h) * (U_e w h)). Scores are the sigmoid (or softmax) of fp32 router logits, the chosen scores are the
    weights.

    ``forward`` returns (rows z, row of every (token, slot), experts per token): the caller adds a token's rows up together
    with the residual. bf16 models run mat-vecs on a few rows, then the grouped tensor-core GEMMs, with the token tile chosen
    from the number of rows per expert; fp32 models and sizes that cannot be copied in 16-byte pieces a row kernel. No step waits for the host."""

    SCORE, RENORM = "sigmoid", False
    GEMV_ROWS, GEMV_PAIRS = 2, 128     # rows per expert and (token, slot) pairs up to which products are mat-vecs
    FEW = 128                  # rows per expert up to which the weights are streamed through the narrow-tile kernel

    @classmethod
    def check(cls, m: dict, index: int) -> None:
        r = m["router"]
        if not 1 <= r["top"] <= min(r["experts"], 16) or r["experts"] > 1024:
            raise ValueError(f"layer {index}: top must lie between 1 and the number of experts (at most 16 of 1024)")

    def __init__(self, m: dict, width: int, dtype, device):
        super().__init__()
        self.E, self.k, self.ff, self.width = m["router"]["experts"], m["router"]["top"], m["expert"]["ff"], width
        new = lambda *s: nn.Parameter(torch.zeros(*s, dtype=dtype, device=device), requires_grad=False)      # noqa: E731
        self.router = new(-(-self.E // 8) * 8, width)
        self.gate_up = new(self.E, 2 * self.ff, width)
        self.down = new(self.E, width, self.ff)

    def named_weights(self):
        f, w = self.ff, self.width
        for e in range(self.E):
            gu, dn = self.gate_up[e], self.down[e]
            yield f"e{e}.gate", (f, w), gu[:f].copy_, lambda gu=gu: gu[:f]
            yield f"e{e}.up", (f, w), gu[f:].copy_, lambda gu=gu: gu[f:]
            yield f"e{e}.down", (w, f), dn.copy_, lambda dn=dn: dn
        yield "router", (self.E, w), self.router[:self.E].copy_, lambda: self.router[:self.E]

    def forward(self, h: torch.Tensor):
        from ..ops import functional as ops
        from ..ops import native as nat
        r = nat.moe_route(ops.router_logits(h, self.router, self.E), self.k, self.RENORM, score=self.SCORE)
        T, f, w = h.shape[0], self.ff, self.width
        if h.dtype != torch.bfloat16 or f % 8 or w % 8:
            xs, off, dest = nat.expert_gather(h, r, self.k)
            return nat.expert_rows(nat.expert_rows(xs, self.gate_up, off, "swiglu"), self.down, off), dest, self.k
        per = -(-T * self.k // self.E)                     # rows of an expert on average
        if per <= self.GEMV_ROWS and T * self.k <= self.GEMV_PAIRS:
            act = nat.expert_gemv(h, self.gate_up, r, self.k, "swiglu")
            return nat.expert_gemv(act, self.down, r, self.k, "none"), r["inv"], self.k
        if per <= self.FEW:
            xs, off, dest = nat.expert_gather(h, r, self.k)
            tile = min(T, 2 * per)
            act = nat.grouped_gemm_skinny(xs, self.gate_up, off, swiglu=True, max_rows_per_expert=tile)
            return nat.grouped_gemm_skinny(act, self.down, off, max_rows_per_expert=tile), dest, self.k
        xs, off, dest = nat.expert_gather(h, r, self.k, align=128)
        gu = nat.grouped_gemm(0, xs, self.gate_up, off, 2 * f, w)
        act = nat.clamped_glu(gu, f, float("inf"), 1.0, 0.0)                        # silu(gate) * up
        return nat.grouped_gemm(0, act, self.down, off, w, f), dest, self.k


class WeightedOutputExperts(nn.Module):
    """Routed experts for serving without a gated unit, down_e(gelu(U_e h)), whose routing weight multiplies the expert's output,
    beside a shared expert that every token uses. Scores are the softmax of fp32 router logits. The choice goes by score +
    correction within the best groups of neighbours; the weights are the scores times a factor. The last ``identity`` router
    outputs stand for h itself.

    ``forward`` returns the summands of ``native.add_normed``, which adds a token's rows up, norms the sum and adds it to the
    stream. The products take the paths of ``WeightedInputExperts``; pairs that chose an identity lie behind the experts' rows and
    are not computed."""

    GEMV_ROWS, GEMV_PAIRS, FEW = WeightedInputExperts.GEMV_ROWS, WeightedInputExperts.GEMV_PAIRS, WeightedInputExperts.FEW

    @classmethod
    def check(cls, m: dict, index: int) -> None:
        r = m["router"]
        n, groups = r["experts"] + r.get("identity", 0), r.get("groups") or {"count": 1, "keep": 1}
        if r["experts"] < 1 or r.get("identity", 0) < 0 or not 1 <= r["top"] <= min(n, 16) or n > 1024:
            raise ValueError(f"layer {index}: top must lie between 1 and the number of experts (at most 16 of 1024)")
        if not 1 <= groups["keep"] <= groups["count"] <= 32 or n % groups["count"] or groups["keep"] * (n // groups["count"]) < r["top"]:
            raise ValueError(f"layer {index}: {n} experts in {groups['count']} groups, of which {groups['keep']} are open to {r['top']} choices")

    def __init__(self, m: dict, width: int, dtype, device):
        super().__init__()
        r = m["router"]
        self.E, self.identity, self.k, self.ff, self.width = r["experts"], r.get("identity", 0), r["top"], m["expert"]["ff"], width
        groups = r.get("groups") or {"count": 1, "keep": 1}
        self.groups, self.keep, self.factor = groups["count"], groups["keep"], float(r.get("scale", 1.0))
        self.shared_ff = m["shared"]["ff"] if m.get("shared") else 0
        up8 = lambda n: -(-n // 8) * 8      # noqa: E731
        new = lambda *s: nn.Parameter(torch.zeros(*s, dtype=dtype, device=device), requires_grad=False)      # noqa: E731
        self.router = new(up8(self.E + self.identity), width)
        self.correction = nn.Parameter(torch.zeros(self.E + self.identity, device=device), requires_grad=False)
        self.up, self.down = new(self.E, self.ff, width), new(self.E, width, self.ff)
        if self.shared_ff:
            self.shared_up, self.shared_down = new(up8(self.shared_ff), width), new(up8(width), self.shared_ff)

    def named_weights(self):
        f, w, n, s = self.ff, self.width, self.E + self.identity, self.shared_ff
        for e in range(self.E):
            up, dn = self.up[e], self.down[e]
            yield f"e{e}.up", (f, w), up.copy_, lambda up=up: up
            yield f"e{e}.down", (w, f), dn.copy_, lambda dn=dn: dn
        yield "router", (n, w), self.router[:n].copy_, lambda: self.router[:n]
        yield "correction", (n,), self.correction.copy_, lambda: self.correction
        if s:
            yield "shared.up", (s, w), self.shared_up[:s].copy_, lambda: self.shared_up[:s]
            yield "shared.down", (w, s), self.shared_down[:w].copy_, lambda: self.shared_down[:w]

    def _shared(self, h: torch.Tensor) -> torch.Tensor:
        from ..ops import functional as ops
        from ..ops import native as nat
        if h.dtype == torch.bfloat16 and ops.gemv_fits(*h.shape) and h.stride(0) % 8 == 0:
            a = nat.gemv_ex(h, self.shared_up, n=self.shared_ff, gelu=True)
        else:
            a = ops.project(h, self.shared_up)
            a = nat.gelu(a, a)[:, :self.shared_ff]
        return ops.project(a, self.shared_down)

    def _routed(self, h: torch.Tensor, r: dict):
        """(expert rows, row of every (token, slot))."""
        from ..ops import native as nat
        T, f, w, k = h.shape[0], self.ff, self.width, self.k
        if h.dtype != torch.bfloat16 or f % 8 or w % 8:
            xs, off, dest = nat.expert_gather(h, r, k, weighted=False)
            return nat.expert_rows(nat.expert_rows(xs, self.up, off, "gelu"), self.down, off), dest
        per = -(-T * k // self.E)                          # rows of an expert on average
        if per <= self.GEMV_ROWS and T * k <= self.GEMV_PAIRS:
            return nat.expert_gemv(nat.expert_gemv(h, self.up, r, k, "gelu"), self.down, r, k, "none"), r["inv"]
        if per <= self.FEW:
            xs, off, dest = nat.expert_gather(h, r, k, weighted=False)
            tile = min(T, 2 * per)
            act = nat.grouped_gemm_skinny(xs, self.up, off, max_rows_per_expert=tile, gelu=True)
            return nat.grouped_gemm_skinny(act, self.down, off, max_rows_per_expert=tile), dest
        xs, off, dest = nat.expert_gather(h, r, k, align=128, weighted=False)
        return nat.grouped_gemm(0, nat.grouped_gemm(0, xs, self.up, off, f, w, gelu=True), self.down, off, w, f), dest

    def forward(self, h: torch.Tensor) -> dict:
        from ..ops import functional as ops
        from ..ops import native as nat
        r = nat.moe_route(ops.router_logits(h, self.router, self.E + self.identity), self.k, False,
                          choice=(self.correction, self.groups, self.keep, self.factor))
        z, row = self._routed(h, dict(r, counts=r["counts"][:self.E], offsets=r["offsets"][:self.E + 1]))
        return dict(y=self._shared(h) if self.shared_ff else None, z=z, route=(r["topk_w"], r["topk_idx"], row, self.E), k=self.k)


class SparseMoeBlock(nn.Module):
    def __init__(self, cfg: ModelArgs, dtype, device):
        super().__init__()
        self.cfg = cfg
        E, H, I = cfg.num_experts, cfg.hidden_size, cfg.moe_intermediate_size
        self.router = nn.Parameter(torch.empty(E, H, dtype=dtype, device=device))
        self.gate_up = nn.Parameter(torch.empty(E, 2 * I, H, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.empty(E, H, I, dtype=dtype, device=device))
        self.ep_group = None       # set by parallel.ep.shard_experts
        self.local_experts: Optional[Tuple[int, int]] = None

    def forward(self, x: torch.Tensor, residual: Optional[torch.Tensor] = None) -> torch.Tensor:
        cfg = self.cfg
        if getattr(self, "tp_reduce", None) is not None and self.local_experts is not None:
            from ..parallel.tp_model import moe_local_forward
            return moe_local_forward(self, x, residual)      # replicated tokens, this rank's experts, summed over ranks
        logits = F.linear(x, self.router)
        eng = getattr(self, "ep_engine", None)
        if eng is not None and x.is_cuda and not torch.is_grad_enabled() and x.shape[0] * eng.k <= eng.max_rows:
            # fused routing + (expert-parallel) dispatch + grouped GEMMs + combine (parallel/ep.py)
            if residual is not None and x.dtype == torch.bfloat16:
                return eng.forward(x, logits, residual)          # residual add fused into the combine kernel
            out = eng.forward(x.to(torch.bfloat16), logits).to(x.dtype)
            return out if residual is None else out + residual
        w, idx = route_topk(logits, cfg.num_experts_per_tok, cfg.norm_topk_prob)
        if getattr(self, "offload", None) is not None:
            from .expert_store import offloaded_experts_forward
            out = offloaded_experts_forward(self, x, w, idx)     # experts read from a packed directory on demand
        elif self.ep_group is not None and getattr(self, "ep_train", False):
            from ..parallel.ep_train import ep_moe_train_forward
            out = ep_moe_train_forward(self, x, w, idx)          # sharded expert parameters, differentiable exchange
        elif self.ep_group is not None:
            from ..parallel.ep import ep_moe_forward_nccl
            out = ep_moe_forward_nccl(self, x, w, idx)
        else:
            out = self.experts_forward(x, w, idx)
        return out if residual is None else out + residual

    def experts_forward(self, x: torch.Tensor, w: torch.Tensor, idx: torch.Tensor) -> torch.Tensor:
        from ..ops import functional as ops
        return ops.moe_experts(x, w, idx, self.gate_up, self.down)

    def hf_state_dict(self) -> Dict[str, torch.Tensor]:
        if getattr(self, "offload", None) is not None:
            raise RuntimeError("the experts of this block live in a packed directory and cannot be exported from here")
        I = self.cfg.moe_intermediate_size
        sd = {"gate.weight": self.router.detach()}
        for e in range(self.cfg.num_experts):
            sd[f"experts.{e}.gate_proj.weight"] = self.gate_up.detach()[e, :I]
            sd[f"experts.{e}.up_proj.weight"] = self.gate_up.detach()[e, I:]
            sd[f"experts.{e}.down_proj.weight"] = self.down.detach()[e]
        return sd

    @torch.no_grad()
    def load_hf_state_dict(self, sd, prefix: str, strict: bool = True) -> Set[str]:
        used = set()
        I = self.cfg.moe_intermediate_size

        def take(name, dst):
            if name in sd:
                dst.copy_(sd[name].to(dst.dtype))
                used.add(name)
            elif strict:
                raise KeyError(name)
        take(prefix + "gate.weight", self.router)
        if prefix + "switch_mlp.gate_proj.weight" in sd:       # stacked layout used by the reference loader
            self.gate_up[:, :I].copy_(sd[prefix + "switch_mlp.gate_proj.weight"])
            self.gate_up[:, I:].copy_(sd[prefix + "switch_mlp.up_proj.weight"])
            self.down.copy_(sd[prefix + "switch_mlp.down_proj.weight"])
            used |= {prefix + f"switch_mlp.{n}_proj.weight" for n in ("gate", "up", "down")}
            return used
        for e in range(self.cfg.num_experts):
            take(prefix + f"experts.{e}.gate_proj.weight", self.gate_up[e, :I])
            take(prefix + f"experts.{e}.up_proj.weight", self.gate_up[e, I:])
            take(prefix + f"experts.{e}.down_proj.weight", self.down[e])
        return used
