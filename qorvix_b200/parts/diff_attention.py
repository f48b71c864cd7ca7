"""Differential attention over the paged cache: two softmax maps per head over one set of values, the second
subtracted from the first times a number of the layer, the difference unit-normed per head.  q, k and v come from
one fused projection with float32 sums; one kernel adds the biases, norms and rotates every map of q and k (each where the
model has it) and writes k and v into the token's cache row (keys of both maps, then values); attention reads keys and values
from the pages only, so a prompt portion and a single decoded token take the same path.  Where a model has none of the
three, the projection leaves in the compute type, its query columns are read where they lie and its other columns are
the token's cache row.
"""
from __future__ import annotations

import math

import torch

from ..cache.spec import PagedRowsSpec
from ..csrc import ops
from .base import Mixer
from .linear import Linear
from .registry import build_part, register_part


class DiffAttention(Mixer):
    def __init__(self, spec, source, rt):
        self.spec, self.rt = spec, rt
        self.H, self.G, self.n, self.dv = spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim
        if self.H % self.G:
            raise ValueError(f"num_heads {self.H} is not a multiple of num_kv_heads {self.G}")
        mats = [source.get(spec.q_proj), source.get(spec.k_proj), source.get(spec.v_proj)]
        dt = torch.float32 if any(m.dtype == torch.float32 for m in mats) else mats[0].dtype
        has_bias = getattr(spec, "bias", True)
        if (spec.q_norm is None) != (spec.k_norm is None):
            raise ValueError("differential attention norms both q and k or neither")
        self.plain = not has_bias and spec.q_norm is None and spec.position is None
        rows = sum(m.shape[0] for m in mats)
        if self.plain and dt == torch.bfloat16 and rows % 8:
            mats.append(torch.zeros((-rows) % 8, mats[0].shape[1], device=mats[0].device, dtype=dt))     # every token's row starts on 16 bytes
        self.qkv_proj = Linear(torch.cat([m.to(dt) for m in mats], dim=0))
        del mats
        self.bias = (torch.cat([source.get(name + ".b", dtype=torch.float32) for name in (spec.q_proj, spec.k_proj, spec.v_proj)]).contiguous()
                     if has_bias else None)
        self.q_weight = source.get(spec.q_norm, dtype=torch.float32) if spec.q_norm is not None else None
        self.k_weight = source.get(spec.k_norm, dtype=torch.float32) if spec.k_norm is not None else None
        lq1, lk1, lq2, lk2 = (source.get(name, dtype=torch.float64).cpu() for name in (spec.lam_q1, spec.lam_k1, spec.lam_q2, spec.lam_k2))
        # one number a layer, formed once on the host
        self.lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + float(spec.diff)
        self.o_proj = Linear(source.get(spec.o_proj))
        self.position = build_part("position", spec.position, source, rt)
        self.rot = int(spec.position.rotary_dim) if spec.position is not None else 0
        self.window = int(spec.window)

    def cache_spec(self):
        return PagedRowsSpec(self.G * (2 * self.n + self.dv), self.window)

    def forward(self, x, ctx, cache):
        s, H, G, n, dv = self.spec, self.H, self.G, self.n, self.dv
        T = x.shape[0]
        bt = ctx.block_tables[cache.group]
        if self.plain:
            proj = self.qkv_proj(x, out_dtype=self.rt.dtype)
            q = proj[:, : H * 2 * n]
            ops.cache_rows(cache.tensor, proj[:, H * 2 * n: (H + G) * 2 * n + G * dv], ctx, bt, cache.page_size)
        else:
            proj = self.qkv_proj(x, out_dtype=torch.float32)
            q = torch.empty((T, H * 2 * n), device=x.device, dtype=self.rt.dtype)
            table = self.position.table() if self.position is not None else None
            ops.diff_prepare(q, proj, self.bias, self.q_weight, self.k_weight, s.eps, table, ctx, bt, cache.tensor, H, G, n, dv, self.rot,
                             cache.page_size)
        out = torch.empty((T, H * dv), device=x.device, dtype=self.rt.dtype)
        ops.diff_attention(out, q, cache.tensor, ctx, bt, H, G, n, dv, cache.page_size, self.window, s.scale, self.lam, s.eps,
                           1.0 - float(s.diff))
        return self.o_proj(out, out_dtype=self.rt.dtype)


register_part("mixer", "diff_attention", DiffAttention)
