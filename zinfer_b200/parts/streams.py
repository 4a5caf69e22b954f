"""Residual streams (hyper-connections): several rows per token instead of one.

The rows between a model's embedding and its final norm are x [S, tokens, width], float32, every stream the embedding's
row at the start.  A sublayer reads one learned combination of the streams and writes back into all of them:

    u = sum_s read[s] x_s        y = sublayer(norm(u))        x_t <- sum_s mix[s, t] x_s + out[t] y   (all t from the old x)

`StreamNorm` is the norm of such a combination (of the plain sum, without a `read_name`: the final norm); `StreamBlock` is
the block of a mixer and a feed-forward, each with a read, a mix and an out vector of its own.  The pass that writes the
streams back also makes the normalised row that the NEXT sublayer reads (`kernels.stream_step`), within a block and, through
`forward_chained`, from one block to the next and to the final norm, so a sublayer costs one pass over the streams."""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from .base import BLOCKS, NORMS, Block, FeedForward, Mixer, Norm, WeightSpec


class PreparedRows:
    """The rows `norm` makes of the streams as they now are, made by the pass that wrote the streams."""

    def __init__(self, norm: "StreamNorm", rows: torch.Tensor):
        self.norm, self.rows = norm, rows


class StreamNorm(Norm):
    """RMS norm of sum_s read[s] x_s; `one_plus`: the weight is stored around zero and 1 + w multiplies."""

    def __init__(self, dim: int, eps: float, weight_name: str, streams: int, read_name: Optional[str] = None,
                 one_plus: bool = False):
        self.dim, self.eps, self.streams, self.one_plus = dim, float(eps), int(streams), bool(one_plus)
        self.weight_name, self.read_name = weight_name, read_name
        self.weight = self.read = None

    def weight_specs(self):
        specs = [WeightSpec(self.weight_name, (self.dim,), role="vector", init="normal" if self.one_plus else "norm")]
        if self.read_name is not None:
            specs.append(WeightSpec(self.read_name, (self.streams,), role="vector", init="norm"))
        return specs

    def load(self, weights, dtype, device):
        if self.streams > kernels.stream_max():
            raise ValueError(f"{self.streams} residual streams; the kernels take at most {kernels.stream_max()}")
        w = weights[self.weight_name]
        self.weight = w + 1.0 if self.one_plus else w
        self.read = weights[self.read_name] if self.read_name is not None else None

    def forward(self, ctx, x, rows=None):
        return kernels.stream_norm(x, self.read, self.weight, self.eps, ctx.dtype, rows)

    def pending(self, ctx, x, prepared=None):
        """The prepared rows if the streams' last pass made them for this norm; nothing is left pending otherwise."""
        return prepared.rows if isinstance(prepared, PreparedRows) and prepared.norm is self else None


class StreamBlock(Block):
    def __init__(self, mixer_norm: StreamNorm, mixer: Mixer, mixer_write: tuple[str, str],
                 ffn_norm: Optional[StreamNorm] = None, ffn: Optional[FeedForward] = None,
                 ffn_write: Optional[tuple[str, str]] = None):
        """mixer_write, ffn_write: the names of (mix [S, S], out [S]) of that sublayer.  `ffn` None: the mixer alone."""
        if not (ffn is None) == (ffn_norm is None) == (ffn_write is None):
            raise ValueError("a feed-forward, its norm and its stream weights come together")
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn = mixer_norm, mixer, ffn_norm, ffn
        self.mixer_write, self.ffn_write = mixer_write, ffn_write
        self.streams = mixer_norm.streams
        self.mixer_mix = self.mixer_out = self.ffn_mix = self.ffn_out = None

    def parts(self):
        return [p for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if p is not None]

    def weight_specs(self):
        S = self.streams
        return [WeightSpec(name, shape, role="vector", init="norm" if len(shape) == 1 else "normal")
                for pair in (self.mixer_write, self.ffn_write) if pair is not None
                for name, shape in zip(pair, ((S, S), (S,)))]

    def load(self, weights, dtype, device):
        self.mixer_mix, self.mixer_out = (weights[n] for n in self.mixer_write)
        if self.ffn_write is not None:
            self.ffn_mix, self.ffn_out = (weights[n] for n in self.ffn_write)

    def entry_norm(self):
        return self.mixer_norm

    def forward(self, ctx, call, x):
        self.forward_chained(ctx, call, x)

    @staticmethod
    def _read(norm, ctx, x, prepared):
        h = norm.pending(ctx, x, prepared)
        return norm.forward(ctx, x) if h is None else h

    @staticmethod
    def _write(ctx, x, y, mix, out, next_norm) -> Optional[PreparedRows]:
        if not isinstance(next_norm, StreamNorm):
            kernels.stream_step(x, y, mix, out)
            return None
        return PreparedRows(next_norm, kernels.stream_step(x, y, mix, out, next_norm.read, next_norm.weight, next_norm.eps, ctx.dtype))

    def forward_chained(self, ctx, call, x, entry=None, next_norm=None):
        y = torch.empty_like(x[0])
        self.mixer.forward(ctx, call, self._read(self.mixer_norm, ctx, x, entry), y, False)
        made = self._write(ctx, x, y, self.mixer_mix, self.mixer_out, next_norm if self.ffn is None else self.ffn_norm)
        if self.ffn is None:
            return made
        self.ffn.forward(ctx, self._read(self.ffn_norm, ctx, x, made), y, False)
        return self._write(ctx, x, y, self.ffn_mix, self.ffn_out, next_norm)


NORMS.register("stream_rmsnorm", StreamNorm)
BLOCKS.register("streams", StreamBlock)
