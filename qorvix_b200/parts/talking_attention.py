"""Causal grouped-query attention whose heads talk: rotated queries and keys, soft-capped scores, a sink in every head's
softmax, and the heads' weights mixed by a matrix before they meet the values; values may be shared between layers.  q, k
and v are one fused product with float32 sums; the preparing kernel (csrc/bias_attention.cu, `rot_norm_prepare` without the unit
norm) rotates in float32, blends the values with the sharing layer's where asked, writes q in the compute type and k and v
into the token's cache row [keys of all key/value heads | their values]; attention is csrc/talking_attention.cu."""
from __future__ import annotations

import torch

from ..cache.spec import PagedRowsSpec
from ..csrc import ops
from .base import Mixer
from .linear import Linear
from .registry import build_part, register_part
from .shared_io import stack_rows


class TalkingAttention(Mixer):
    def __init__(self, spec, source, rt):
        self.spec, self.rt = spec, rt
        self.H, self.G, self.n, self.dv = spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim
        if self.H % self.G:
            raise ValueError(f"num_heads {self.H} is not a multiple of num_kv_heads {self.G}")
        self.qkv = Linear(stack_rows([source.get(spec.q_proj), source.get(spec.k_proj), source.get(spec.v_proj)]))
        self.o_proj = Linear(source.get(spec.o_proj))
        self.position = build_part("position", spec.position, source, rt)
        self.table = self.position.table() if self.position is not None else None
        if self.position is not None and self.table is None:
            raise ValueError("this attention rotates from a cos/sin table: its position must be a rotary encoding")
        self.rot = self.table.shape[1] * 2 if self.table is not None else 0
        self.interleaved = getattr(spec.position, "pairing", "split_half") == "interleaved"
        self.sink = source.get(spec.sink, dtype=torch.float32).reshape(-1).contiguous()
        self.talk = source.get(spec.talk, dtype=torch.float32).contiguous()
        self.talk_host = self.talk.cpu().contiguous()
        self.role = spec.v_share_role
        if self.role not in (None, "source", "blend"):
            raise ValueError(f"unknown role '{self.role}' in value sharing (known: source, blend)")
        if self.role is not None and not spec.v_share:
            raise ValueError("a layer that shares values names what it shares (v_share)")
        self.lam = float(source.get(spec.v_blend, dtype=torch.float32).item()) if self.role == "blend" else 0.0

    def cache_spec(self):
        return PagedRowsSpec(self.G * (self.n + self.dv), 0)

    def forward(self, x, ctx, cache):
        H, G, n, dv = self.H, self.G, self.n, self.dv
        bt = ctx.block_tables[cache.group]
        proj = self.qkv(x, out_dtype=torch.float32)
        k_off, v_off = H * n, (H + G) * n
        v_other = None
        if self.role == "source":
            ctx.shared[self.spec.v_share] = proj[:, v_off: v_off + G * dv]
        elif self.role == "blend":
            v_other = ctx.shared.get(self.spec.v_share)
            if v_other is None or tuple(v_other.shape) != (proj.shape[0], G * dv):
                raise ValueError(f"no layer ahead of this one has left values of {G} x {dv} under '{self.spec.v_share}'")
        q = torch.empty((proj.shape[0], H * n), device=proj.device, dtype=self.rt.dtype)
        ops.rot_norm_prepare(q, proj, 0, k_off, v_off, cache.tensor, self.table, self.rot, False, 0.0, None, v_other, self.lam, ctx, bt, H, G, n,
                             dv, cache.page_size, interleaved=self.interleaved)
        out = torch.empty((proj.shape[0], H * dv), device=proj.device, dtype=self.rt.dtype)
        ops.talking_attention(out, q, cache.tensor, ctx, bt, H, G, n, dv, cache.page_size, float(self.spec.scale), float(self.spec.softcap),
                              self.sink, self.talk, self.talk_host)
        return self.o_proj(out, out_dtype=self.rt.dtype)


register_part("mixer", "talking_attention", TalkingAttention)
