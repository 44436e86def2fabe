"""Differential attention: the difference of two softmax maps over the same values."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np
import torch

from ..cache.manager import CacheNeed
from ..kernels import ops
from ..weights.tensor_spec import TensorSpec
from .base import LayerCache, Mixer, register_part
from .scaled_attention import attend

MAPS = 2


def query_temperature_table(coef: float, every: float, length: int) -> np.ndarray:
    """[length] float32: 1 + coef * ln(floor((p + 1) / every) + 1) at position p; 64-bit, rounded once."""
    p = np.arange(length, dtype=np.float64)
    return (1.0 + coef * np.log(np.floor((p + 1.0) / every) + 1.0)).astype(np.float32)


@register_part("mixer", "difference_attention")
class DifferenceAttention(Mixer):
    """Every query head has two queries and every key/value head two keys, `dim` wide and side by side, and
    one value of `vdim`; query head h reads key/value head h // (heads / kv_heads).  With a_1 and a_2 the
    results of two causal softmax attentions, query m over key m, scores (q . k) * scale:

        o = a_1 - lambda a_2,   lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
        o <- o / sqrt(mean(o^2) + eps) * (1 - diff) * sigmoid(W_g y)[head]

    and the heads pass the output projection.  No positions, no biases; with `temperature` = (coef, every)
    the query at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1) - by a table of
    factors on its scores, in 32-bit.

    The two keys of a head are one row of the cache, twice as wide, beside one value row.  The kernels
    of the scaled attention run both maps over the one tile of values they have fetched; what they leave of
    every key range is merged, subtracted, normed and gated by one kernel, in 32-bit (`difference_merge`).
    W_g rides in the one product with q, k and v.  `names` gives the tensor names below the prefix.
    """

    capturable = True

    NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "o": "o", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2",
             "lk2": "lk2"}

    def __init__(self, prefix: str, hidden_size: int, heads: int, kv_heads: int, dim: int, vdim: int,
                 scale: float, diff: float, eps: float, temperature: Optional[tuple] = None,
                 names: Optional[Dict[str, str]] = None):
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        self.prefix, self.hidden_size = prefix, int(hidden_size)
        self.heads, self.kv_heads, self.dim, self.vdim = int(heads), int(kv_heads), int(dim), int(vdim)
        self.scale, self.diff, self.eps = float(scale), float(diff), float(eps)
        self.temperature = None if temperature is None else (float(temperature[0]), float(temperature[1]))
        if self.vdim > 512:
            raise ValueError(f"difference_attention: values {self.vdim} wide, the kernels hold 512")
        self.q_width, self.k_width = self.heads * MAPS * self.dim, self.kv_heads * MAPS * self.dim
        self.v_width = self.kv_heads * self.vdim
        self.names = dict(self.NAMES)
        self.names.update(names or {})
        self.w_in = self.w_o = self.head_scale = self.no_table = self.pos_scale = None
        self.weight = 0.0

    def tensor_specs(self) -> List[TensorSpec]:
        p, h, n = self.prefix, self.hidden_size, self.names
        return [TensorSpec(p + n["q"], (self.q_width, h)), TensorSpec(p + n["k"], (self.k_width, h)),
                TensorSpec(p + n["v"], (self.v_width, h)), TensorSpec(p + n["gate"], (self.heads, h)),
                TensorSpec(p + n["o"], (h, self.heads * self.vdim))] + \
            [TensorSpec(p + n[which], (self.dim,), role="vector") for which in ("lq1", "lk1", "lq2", "lk2")]

    def cache_need(self) -> Optional[CacheNeed]:
        wide = MAPS * self.dim
        return CacheNeed(self.kv_heads, wide, 0, 0, 0 if self.vdim == wide else self.vdim)

    def bind(self, tensors: Dict[str, torch.Tensor], runtime) -> None:
        self.runtime = runtime
        p, n = self.prefix, self.names
        stacked = [tensors[p + n[which]] for which in ("q", "k", "v", "gate")]
        rows = sum(w.shape[0] for w in stacked)
        if rows % 8:                        # rows of the product's result start on 16 bytes
            stacked.append(torch.zeros(8 - rows % 8, self.hidden_size, dtype=stacked[0].dtype, device=stacked[0].device))
        self.w_in = torch.cat(stacked).contiguous()
        self.w_o = tensors[p + n["o"]].contiguous()
        a, b, c, d = (tensors[p + n[which]].double() for which in ("lq1", "lk1", "lq2", "lk2"))
        self.weight = math.exp(float((a * b).sum())) - math.exp(float((c * d).sum())) + self.diff
        self.head_scale = torch.full((self.heads * MAPS,), self.scale, dtype=torch.float32, device=runtime.device)
        self.no_table = runtime.shared_table(("rotary-none",), lambda: torch.zeros((1, 0), dtype=torch.float32))
        if self.temperature is not None:
            length = max(runtime.max_positions, 1)
            self.pos_scale = runtime.shared_table(
                ("query_temperature", *self.temperature, length),
                lambda: torch.from_numpy(query_temperature_table(*self.temperature, length)))
        runtime.prepare_weight(self.w_in)
        runtime.prepare_weight(self.w_o)

    def forward(self, ctx, y: torch.Tensor, cache: LayerCache) -> torch.Tensor:
        rt = self.runtime
        tokens, wide = y.shape[0], MAPS * self.dim
        group = ctx.groups[cache.group]
        proj = rt.linear(y, self.w_in, None, "difference_attention.in")
        # keys and values into their pages (nothing to norm or rotate: the queries stay as they are)
        ops.norm_rotate_write(proj, ctx.positions, self.no_table, group.slot_of, cache.k_pages, cache.v_pages,
                              cache.page_stride, group.page_size, self.heads, self.kv_heads, wide, self.vdim, 0, None,
                              None, self.eps, ctx.error)
        out = rt.buffer("difference_attention.out", tokens, self.heads * self.vdim, proj.dtype)
        gate0 = self.q_width + self.k_width + self.v_width
        gate = proj[:, gate0:gate0 + self.heads]

        def merge(part_o, part_ml, ranges, listed, count):
            ops.difference_merge(part_o, part_ml, out, tokens, self.heads, self.vdim, ranges, self.weight, self.eps,
                                 1.0 - self.diff, gate, listed, count)
        attend(ctx, rt, proj, self.head_scale, group, cache, out, self.heads * MAPS, self.kv_heads, wide, self.vdim,
               False, 0, pos_scale=self.pos_scale, maps=MAPS, merge=merge)
        return rt.linear(out, self.w_o, None, "difference_attention.o")
