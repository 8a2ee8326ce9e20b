"""Hyper-connections: an arrangement whose residual stream is `streams` copies x_1 .. x_S of the width, side by side in
one 32-bit row per token (all equal to the embedding at the start; the model's end is their sum).  A layer has a norm
before each branch, and per branch three small sets of weights, `in` [S], `mix` [S, S] as [from, to] and `out` [S]:

    u = sum_s in[s] x_s;  y = branch(norm(u));  x_t <- sum_s mix[s, t] x_s + out[t] y      (all t at once)

(a layer without a feed-forward has one branch).  The kernel that updates the streams with a branch's output also forms
what the next branch reads (this layer's or the next one's weighted sum and its norm, or the model's last norm of the
streams' sum), so a branch costs one row-wise launch; it adds a branch's output bias and 32-bit partial sums too.
"""
from __future__ import annotations

from typing import List, Mapping

import torch

from .. import ops
from ..config.base import LayerSpec, PartSpec
from ..errors import SpecError
from ..registry import register_part
from .base import CallStore, Part, Runtime, StepInfo, WeightSpec
from .block import Layer

MAX_STREAMS = 16


class StreamMix(Part):
    """One branch's weights over the streams, kept in 32-bit."""
    graph_safe = True

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.streams = int(spec.params["streams"])
        if not 1 <= self.streams <= MAX_STREAMS:
            raise SpecError(f"arch spec error: {self.streams} residual streams are outside 1..{MAX_STREAMS}")

    def weight_specs(self) -> List[WeightSpec]:
        w, s = self.spec.weights, self.streams
        return [WeightSpec(w["in"], (s,), "vector", 0.5), WeightSpec(w["out"], (s,), "vector", 0.5),
                WeightSpec(w["mix"], (s, s), "vector", 0.5)]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        w = self.spec.weights
        self.w_in, self.w_out, self.w_mix = (self._vector32(tensors[w[r]]) for r in ("in", "out", "mix"))


class StreamNorm:
    """What a branch reads: the norm of a weighted sum of the streams.  Stands where the chain of layers expects the
    next layer's entry norm."""

    def __init__(self, mix: StreamMix, norm):
        self.mix, self.norm = mix, norm

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        s = self.mix.streams
        h = torch.empty((x.shape[0], x.shape[1] // s), dtype=self.norm.rt.dtype, device=x.device)
        ops.hyper_norm(x, s, in_next=self.mix.w_in, w=self.norm.weight, eps=self.norm.eps, h=h)
        return h


class HyperLayer(Layer):
    norm_roles = ("pre_mixer",)
    chains = True

    def __init__(self, spec: LayerSpec, rt: Runtime):
        super().__init__(spec, rt)
        from .feedforward import NoFeedForward
        from .norm import RMSNorm
        self.has_ffn = not isinstance(self.feed_forward, NoFeedForward)
        self.streams = int(spec.params["streams"])
        roles = ("pre_mixer", "pre_ffn") if self.has_ffn else ("pre_mixer",)
        for r in roles:
            if not isinstance(self.norms.get(r), RMSNorm) or self.norms[r].add_one:
                raise SpecError(f"arch spec error: hyper-connections take a plain RMS norm as {r}")
        names = spec.params["mixes"]               # {"mixer": {"in", "out", "mix"}, "ffn": the same}
        self.mixes = [StreamMix(PartSpec("stream_mix", {"streams": self.streams}, names[k]), rt)
                      for k in (("mixer", "ffn") if self.has_ffn else ("mixer",))]
        self._entries = [StreamNorm(m, self.norms[r]) for m, r in zip(self.mixes, roles)]

    def parts(self):
        return super().parts() + self.mixes

    def entry_norm(self):
        return self._entries[0]

    def _update(self, branch, y, x, mix: StreamMix, nxt):
        """The streams with a branch's output, and what `nxt` makes of the new ones."""
        from .norm import RMSNorm
        args = dict(y=y, bias=getattr(branch, "out_bias", None), mix=mix.w_mix, out_w=mix.w_out)
        s = self.streams
        if isinstance(nxt, StreamNorm) or (isinstance(nxt, RMSNorm) and not nxt.add_one):
            norm = nxt.norm if isinstance(nxt, StreamNorm) else nxt
            h = torch.empty((x.shape[0], x.shape[1] // s), dtype=self.rt.dtype, device=x.device)
            ops.hyper_norm(x, s, in_next=nxt.mix.w_in if isinstance(nxt, StreamNorm) else None, w=norm.weight, eps=norm.eps, h=h, **args)
            return h
        ops.hyper_norm(x, s, **args)
        return None

    @staticmethod
    def _run(part, *args):
        """A branch's output without its bias where the branch can leave that to the update."""
        if hasattr(part, "forward_unbiased"):
            return part.forward_unbiased(*args)
        if getattr(part, "out_bias", None) is None and hasattr(part, "forward_partial"):
            return part.forward_partial(*args)
        return part.forward(*args)

    def forward(self, x: torch.Tensor, step: StepInfo, store: CallStore, h_in=None, next_norm=None):
        h = h_in if h_in is not None else self._entries[0].forward(x)
        a = self._run(self.mixer, h, step, store)
        if not self.has_ffn:
            return self._update(self.mixer, a, x, self.mixes[0], next_norm)
        h = self._update(self.mixer, a, x, self.mixes[0], self._entries[1])
        f = self._run(self.feed_forward, h, step)
        return self._update(self.feed_forward, f, x, self.mixes[1], next_norm)


register_part("arrangement", "hyper_prenorm", HyperLayer)
