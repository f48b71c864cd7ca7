"""Gated feed-forward: down(act(gate x) * up x), dense, no bias; act is SiLU
(reference: runtime/src/text_model.cpp:162-168, runtime/src/ops.cpp:96-100) or the tanh form of GELU, or both halves are
clamped first (SwiGLUSpec).  gate and up are one fused projection."""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import FeedForward, PreNormed
from .linear import Linear
from .registry import register_part


GLU_ACTIVATIONS = {"silu": ops.GLU_SILU, "gelu_tanh": ops.GLU_GELU_TANH, "clamped": ops.GLU_CLAMPED}


class SwiGLU(FeedForward):
    def __init__(self, spec, source, rt):
        self.rt = rt
        self.f = int(spec.intermediate_size)
        g, u = source.get(spec.gate_proj), source.get(spec.up_proj)
        dt = torch.float32 if (g.dtype == torch.float32 or u.dtype == torch.float32) else g.dtype
        # When the width allows, gate and up rows are interleaved in groups of 16 (16 gate rows, the 16
        # up rows of the same features, ...), so that one tile of the product holds both halves of a
        # feature and the activation is applied in the product's epilogue.
        acts = GLU_ACTIVATIONS
        name = getattr(spec, "activation", "silu")
        if name not in acts:
            raise ValueError(f"unknown activation '{name}' (known: {', '.join(acts)})")
        self.act = acts[name]
        self.limit, self.slope = float(getattr(spec, "limit", 0.0)), float(getattr(spec, "slope", 0.0))
        self.interleaved = self.f % 16 == 0
        if self.interleaved:
            k = g.shape[1]
            fused = torch.stack([g.to(dt).view(self.f // 16, 16, k), u.to(dt).view(self.f // 16, 16, k)], dim=1)
            self.gate_up = Linear(fused.reshape(2 * self.f, k))
            del fused
        else:
            self.gate_up = Linear(torch.cat([g.to(dt), u.to(dt)], dim=0))
        del g, u
        self.down = Linear(source.get(spec.down_proj))

    folds_norms = True             # forward() takes a PreNormed x, residual= and next_norm=

    def forward(self, x, ctx, residual=None, next_norm=None):
        """x: the normed rows [T, d], or a PreNormed (few tokens: the norm's scale is then applied to the
        gate/up sums before the activation).  With residual and next_norm the down projection adds the
        output to the stream itself and the PreNormed input of next_norm is returned instead."""
        act = None
        if isinstance(x, PreNormed):
            act = torch.empty((x.scaled.shape[0], self.f), device=x.scaled.device, dtype=self.rt.dtype)
            if not (self.interleaved and self.act != ops.GLU_CLAMPED and self.gate_up.forward_prenormed(x, act, swiglu=ops.glu_epilogue(self.act))):
                act, x = None, x.materialise()
        if act is None:
            act = torch.empty((x.shape[0], self.f), device=x.device, dtype=self.rt.dtype)
            if self.interleaved:
                ops.gemm_swiglu(act, x, self.gate_up.weight, self.gate_up.packed, self.gate_up.out_features, act=self.act,
                               limit=self.limit, slope=self.slope)
            else:
                gu = self.gate_up(x, out_dtype=self.rt.dtype)
                ops.glu_act(act, gu, self.act, limit=self.limit, slope=self.slope)
        if residual is not None and next_norm is not None:
            pre = self.down.forward_to_stream(act, residual, next_norm)
            if pre is not None:
                return pre
        return self.down(act, out_dtype=self.rt.dtype)


class ActMLP(FeedForward):
    """Ungated feed-forward: down(act(up x)), the up product's bias, where there is one, and the activation (the square of
    relu, or the tanh form of GELU) in that product's epilogue where the kernel takes it, else a pass of their own; the down product's bias is offered to the block."""

    def __init__(self, spec, source, rt):
        acts = {"relu2": ops.ACT_RELU2, "gelu_tanh": ops.ACT_GELU_TANH}
        if spec.activation not in acts:
            raise ValueError(f"unknown activation '{spec.activation}' (known: {', '.join(acts)})")
        self.act = acts[spec.activation]
        self.rt = rt
        self.up = Linear(source.get(spec.up_proj))
        self.down = Linear(source.get(spec.down_proj))
        bias = getattr(spec, "bias", False)
        self.up_bias = source.get(spec.up_proj + ".b", dtype=torch.float32) if bias else None
        self.output_bias = source.get(spec.down_proj + ".b", dtype=torch.float32) if bias else None

    def forward(self, x, ctx, with_bias: bool = True):
        act = torch.empty((x.shape[0], self.up.out_features), device=x.device, dtype=self.rt.dtype)
        ops.gemm_act(act, x, self.up.weight, self.up.packed, self.up.out_features, self.act, self.up_bias)
        if self.output_bias is None or not with_bias:
            return self.down(act, out_dtype=self.rt.dtype)
        y = self.down(act, out_dtype=torch.float32)
        ops.add_vector(y, self.output_bias)
        return y


register_part("feed_forward", "swiglu", SwiGLU)
register_part("feed_forward", "act_mlp", ActMLP)
