"""A residual stream kept as several copies ("streams") that every sublayer reads and writes through small learned mixtures:

  u = sum_s a_s X_s;   y = sublayer(norm(u));   X_t <- sum_s M[s, t] X_s + b_t y     (all t at once, from the old streams)

with vectors a, b and a matrix M (indexed [from, to]) per sublayer, X [T, streams, hidden] fp32, all streams the embedding at
first and summed in front of the final norm.  The block passes on what the streams have not taken in yet (`StreamDelta`: the
sublayer's result with its M and b), so that one kernel between two sublayers takes the result in, reads the next mixture and
makes its norm."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import Block, FeedForward, Mixer, Norm, Runtime, StepContext, WeightSpec, register_block


class StreamDelta:
    """A sublayer's result that the streams have not taken in yet, with the sublayer's mixing matrix and weights."""
    __slots__ = ("y", "mix", "out_w")

    def __init__(self, y: torch.Tensor, mix: torch.Tensor, out_w: torch.Tensor):
        self.y, self.mix, self.out_w = y, mix, out_w

    def data_ptr(self) -> int:
        return self.y.data_ptr()

    def own_tensors(self) -> List[torch.Tensor]:
        return [self.mix, self.out_w]

    def __iter__(self):
        return iter((self.y, self.mix, self.out_w))


@register_block("mixed_streams")
class MixedStreamsBlock(Block):
    """Pre-norm sublayers between the streams: the mixer with the layer's first set of mixtures, the feed-forward (if there is
    one) with the second.  `names`: the local name prefixes of the two sets; each holds `in` [streams], `out` [streams] and
    `mix` [streams, streams]."""

    def __init__(self, params: dict, rt: Runtime, mixer_norm: Norm, mixer: Mixer, ffn_norm: Norm, feed_forward: FeedForward):
        self.rt = rt
        self.prefix = params.get("prefix", "")
        self.size, self.streams = int(params["size"]), int(params["streams"])
        if not 0 < self.streams <= ops.MAX_STREAMS:
            raise ValueError(f"mixed_streams: {self.streams} streams (at most {ops.MAX_STREAMS})")
        self.mixer_norm, self.mixer, self.ffn_norm, self.feed_forward = mixer_norm, mixer, ffn_norm, feed_forward
        self.has_ff = not getattr(feed_forward, "absent", False)
        names = tuple(params.get("names", ("mixer_streams.", "ffn_streams.")))
        self.names = names if self.has_ff else names[:1]
        self.sets: List[tuple] = []                  # per sublayer: (in [S], mix [S, S], out [S]) fp32
        self.ones = torch.ones((self.streams,), dtype=torch.float32, device=rt.device)       # the plain sum of the streams

    def weight_specs(self) -> Dict[str, WeightSpec]:
        S, specs = self.streams, {}
        for n in self.names:
            specs[n + "in"] = WeightSpec((S,), role="vector", init=("normal", 0.7))
            specs[n + "out"] = WeightSpec((S,), role="vector", init=("one_plus_normal", 0.3))
            specs[n + "mix"] = WeightSpec((S, S), role="vector", init=("normal", 0.7))
        return specs

    def kernel_sources(self):
        return [("streams.cu", {})]

    def bind(self, tensors):
        self.sets = [(tensors[n + "in"], tensors[n + "mix"], tensors[n + "out"]) for n in self.names]

    def replay_key(self):
        keys = [p.replay_key() for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.feed_forward)]
        return None if any(k is None for k in keys) else ("mixed_streams", self.rt.dtype, self.size, self.streams, *keys)

    def own_tensors(self):
        own = [t for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.feed_forward) for t in p.own_tensors()]
        return own + [t for s in self.sets for t in s]

    def pending(self, delta: StreamDelta) -> StreamDelta:
        """The delta of another layer of equal structure, as this layer's: the same buffer with this layer's mixture."""
        _, mix, out_w = self.sets[-1]
        return StreamDelta(delta.y, mix, out_w)

    def _read(self, streams: torch.Tensor, delta: Optional[StreamDelta], in_w: torch.Tensor, norm: Norm, out: torch.Tensor,
              rows: Optional[torch.Tensor] = None) -> None:
        weight, bias, eps, centred = norm.fused_params()
        ops.streams_mix_norm(streams, delta, in_w, weight, bias, eps, centred, out, rows=rows)

    def forward(self, residual: torch.Tensor, delta: Optional[StreamDelta], ctx: StepContext, cache):
        T = residual.shape[0]
        in_w, mix, out_w = self.sets[0]
        normed = ctx.buffer("block.normed", (T, self.size), self.rt.dtype)
        self._read(residual, delta, in_w, self.mixer_norm, normed)
        delta = StreamDelta(self.mixer.forward(normed, ctx, cache), mix, out_w)
        if self.has_ff:
            in_w, mix, out_w = self.sets[1]
            normed2 = ctx.buffer("block.normed2", (T, self.size), self.rt.dtype)
            self._read(residual, delta, in_w, self.ffn_norm, normed2)
            delta = StreamDelta(self.feed_forward.forward(normed2, ctx), mix, out_w)
        return residual, delta

    # ---- what the model asks of the last block run --------------------------------------------------
    def final_forward(self, residual: torch.Tensor, delta: Optional[StreamDelta], norm: Norm, out: torch.Tensor, rows: torch.Tensor) -> None:
        """out[r] = norm(the sum of the streams at rows[r], the pending result taken in)."""
        self._read(residual, delta, self.ones, norm, out, rows=rows)

    def total(self, residual: torch.Tensor, delta: Optional[StreamDelta]) -> torch.Tensor:
        """The sum of the streams with the pending result taken in, [T, hidden] fp32."""
        out = torch.empty((residual.shape[0], self.size), dtype=torch.float32, device=residual.device)
        ops.streams_total(residual, delta, out)
        return out
