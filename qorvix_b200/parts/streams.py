"""The residual as several streams (hyper-connections).  A sublayer reads a weighted sum of the streams, and its output goes back
to all of them while they are mixed among themselves:
    u = sum_s read[s] x_s;   y = part(norm(u));   x_t <- sum_s mix[s, t] x_s + m * write[t] * y.
The streams lie as one float32 tensor [tokens, streams, width].  A sublayer's output stays pending (a StreamDelta) until the next
sublayer reads: one kernel then writes the streams, sums them for that sublayer and applies its norm, so every stream is read
and written once a sublayer.  All of it is float32.  Ahead of the first write all streams equal the embedding's output, which
is read in their place: nothing is copied."""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import StreamDelta
from .registry import register_part


def read_streams(streams, pending: StreamDelta, read_coef, norm, rt, rows=None):
    """The normed input of a sublayer (norm None: the sum itself, float32) after what is pending has gone back; `rows`: int32 rows to
    read, with nothing stored.  Returns it and what is pending from here on."""
    n = streams.shape[0] if rows is None else rows.numel()
    fused = norm is not None and getattr(norm, "folds_into_products", False) and norm.size == streams.shape[2]
    out = torch.empty((n, streams.shape[2]), device=streams.device, dtype=rt.dtype if fused else torch.float32)
    written = pending.y is not None
    ops.stream_pass(out, streams, read_coef, weight=norm.scale_weight() if fused else None, eps=norm.eps if fused else 0.0,
                    y=pending.y, y_bias=pending.bias, write_coef=pending.link.write_coef if written else None, x0=pending.x0, row_idx=rows,
                    store=written)
    left = StreamDelta() if written and rows is None else pending
    return (out if fused or norm is None else norm.add_norm(out, None)), left


class StreamLink:
    """One sublayer's tie to the streams: what it reads with, and what its output and the old streams go back with."""

    def __init__(self, spec, mult: float, source, rt):
        self.rt = rt
        read, write, mix = (source.get(n, dtype=torch.float32) for n in (spec.read, spec.write, spec.mix))
        self.read_coef = read.contiguous()
        # [mix from/to | write times the multiplier], one small table the kernel takes whole
        self.write_coef = torch.cat([mix.reshape(-1), (write.double() * mult).float()]).contiguous()

    def read(self, streams, pending, norm):
        return read_streams(streams, pending, self.read_coef, norm, self.rt)

    def deliver(self, y, left: StreamDelta, bias=None) -> StreamDelta:
        """The sublayer's output on its way back; `left`: what read() left pending."""
        return StreamDelta(link=self, y=y, bias=bias, x0=left.x0)


class HyperStreams:
    """The streams of a model: where they start and what they end as."""

    def __init__(self, spec, source, rt):
        if not 1 <= spec.count <= ops.MAX_STREAMS:
            raise ValueError(f"{spec.count} residual streams: the kernel takes 1 to {ops.MAX_STREAMS}")
        self.rt, self.count = rt, int(spec.count)
        self.ones = torch.ones(self.count, device=rt.device, dtype=torch.float32)

    def begin(self, x0):
        T, d = x0.shape
        return torch.empty((T, self.count, d), device=x0.device, dtype=torch.float32), StreamDelta(x0=x0)

    def total(self, streams, pending):
        """The sum of the streams after what is pending (float32 [T, d]); nothing is changed."""
        rows = torch.arange(streams.shape[0], device=streams.device, dtype=torch.int32)
        return read_streams(streams, pending, self.ones, None, self.rt, rows=rows)[0]

    def final(self, norm, streams, pending, rows):
        """The normed sum of the streams at the given rows."""
        return read_streams(streams, pending, self.ones, norm, self.rt, rows=rows)[0]


register_part("stream", "hyper_streams", HyperStreams)
