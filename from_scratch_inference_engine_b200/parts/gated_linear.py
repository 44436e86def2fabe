"""Gated linear attention: a recurrence over a matrix per head whose rows decay each at a rate of their own,
token by token."""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from ..weights.tensor_spec import TensorSpec
from .base import LayerCache, Mixer, StateNeed, register_part


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention(Mixer):
    """q = W_q y * dim^(-1/2), k = W_k y [heads, dim]; v = W_v y [heads, vdim]; a decay per key column,
    a = sigmoid(W_a2 (W_a1 y) + b)^(1 / tau) [heads, dim]; per head

        S_t = diag(a_t) S_(t-1) + k_t v_t^T        o_t = S_t^T q_t

    every head of o is divided by its root mean square (`eps` inside the root), multiplied by a gain of vdim
    numbers that all heads share and by silu(W_g y), and the heads pass the output projection.

    The state S [heads, dim, vdim] is float32, zero when a request starts, and lives in the request's
    state slot: a step carries it on from where the last one left it.  Decays (through their logarithms),
    recurrence, norm and gate are 32-bit in both compute dtypes.  q, k, v, the gate and the narrow product
    W_a1 y are one matrix product over the stacked weight; the scan (`ops.lightning_scan` with a decay per
    state row) reads its columns as they are stored.  Prompts of more than two chunks of 64 tokens
    run chunk-parallel.  `rank`, the width of W_a1 y, is the stored tensors' (the parameter is what the
    random-weights mode draws).  `names` gives the tensor names below the prefix.
    """

    capturable = True
    CHUNK_TOKENS = 64

    NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "norm": "norm", "low": "a1", "decay": "a2",
             "decay_bias": "a2.b"}

    def __init__(self, prefix: str, hidden_size: int, heads: int, dim: int, vdim: int, tau: float, eps: float,
                 rank: int = 16, names: Optional[Dict[str, str]] = None):
        self.prefix, self.hidden_size = prefix, int(hidden_size)
        self.heads, self.dim, self.vdim = int(heads), int(dim), int(vdim)
        self.tau, self.eps, self.rank = float(tau), float(eps), int(rank)
        if min(self.heads, self.dim, self.vdim, self.rank) <= 0 or self.tau <= 0:
            raise ValueError("gated_linear_attention: heads, dim, vdim, rank and tau are positive")
        if self.dim > 256:
            raise ValueError(f"gated_linear_attention: {self.dim} state rows per head, the scan holds 256")
        self.qk_width, self.v_width = self.heads * self.dim, self.heads * self.vdim
        self.names = dict(self.NAMES)
        self.names.update(names or {})
        self.w_in = self.w_o = self.gain = self.decay_wt = self.decay_bias = None

    def tensor_specs(self) -> List[TensorSpec]:
        p, h, n = self.prefix, self.hidden_size, self.names
        return [TensorSpec(p + n["q"], (self.qk_width, h)), TensorSpec(p + n["k"], (self.qk_width, h)),
                TensorSpec(p + n["v"], (self.v_width, h)), TensorSpec(p + n["gate"], (self.v_width, h)),
                TensorSpec(p + n["o"], (h, self.v_width)),
                TensorSpec(p + n["norm"], (self.vdim,), role="vector", init="gain"),
                TensorSpec(p + n["low"], (self.rank, h), free=(0,)),
                TensorSpec(p + n["decay"], (self.qk_width, self.rank), role="vector", free=(1,)),
                TensorSpec(p + n["decay_bias"], (self.qk_width,), role="vector")]

    def state_need(self) -> Optional[StateNeed]:
        return StateNeed((self.heads, self.dim, self.vdim), torch.float32)

    def bind(self, tensors: Dict[str, torch.Tensor], runtime) -> None:
        self.runtime = runtime
        p, n = self.prefix, self.names
        low, decay = tensors[p + n["low"]], tensors[p + n["decay"]]
        if low.shape[0] != decay.shape[1]:
            raise ValueError(f"{p}{n['low']} has {low.shape[0]} rows, {p}{n['decay']} {decay.shape[1]} columns")
        self.rank = low.shape[0]
        stacked = [tensors[p + n[which]] for which in ("q", "k", "v", "gate")] + [low]
        rows = sum(w.shape[0] for w in stacked)
        if rows % 8:                        # rows of the product's result start on 16 bytes
            stacked.append(torch.zeros(8 - rows % 8, self.hidden_size, dtype=low.dtype, device=low.device))
        self.w_in = torch.cat(stacked).contiguous()
        self.w_o = tensors[p + n["o"]].contiguous()
        self.gain = tensors[p + n["norm"]].to(torch.float32).contiguous()
        self.decay_wt = decay.to(torch.float32).t().contiguous()
        self.decay_bias = tensors[p + n["decay_bias"]].to(torch.float32).contiguous()
        runtime.prepare_weight(self.w_in)
        runtime.prepare_weight(self.w_o)

    def forward(self, ctx, y: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        rt = self.runtime
        tokens = y.shape[0]
        proj = rt.linear(y, self.w_in, None, "gated_linear.in")
        gate0 = 2 * self.qk_width + self.v_width
        decay = ops.row_decay(proj, gate0 + self.v_width, self.rank, self.decay_wt, self.decay_bias, 1.0 / self.tau,
                              rt.buffer("gated_linear.decay", tokens, self.qk_width, torch.float32))
        chunks = {}
        if int(ctx.h_qlen.max()) > 2 * self.CHUNK_TOKENS:
            tiles = ctx.attention_tiles(1, self.CHUNK_TOKENS)
            chunks = dict(seg_item=tiles.item, seg_row0=tiles.row0, num_segs=tiles.count,
                          seg_tokens=self.CHUNK_TOKENS,
                          chunk_states=ctx.scratch("gated_linear.chunk_states",
                                                   tiles.count * self.qk_width * (self.vdim + 1)))
        o = rt.buffer("gated_linear.o", tokens, self.v_width, torch.float32)
        ops.lightning_scan(proj, 0, self.qk_width, 2 * self.qk_width, ctx.item_qstart, ctx.item_qlen, ctx.item_slots,
                           ctx.num_items, cache.state, None, o, self.heads, self.dim, self.vdim, decay_row=decay,
                           out_scale=self.dim ** -0.5, **chunks)
        gated = rt.buffer("gated_linear.gated", tokens, self.v_width, proj.dtype)
        ops.head_norm_silu(o, proj, gate0, self.gain, self.eps, gated, self.heads)
        return rt.linear(gated, self.w_o, None, "gated_linear.out")
