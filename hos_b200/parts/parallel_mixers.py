"""Two (or more) mixers side by side: all read the same rows, and their outputs are added (each times a constant of its
own, the `out_scale` of its spec).

The mixers' input projections are one product and their output projections another: the first one's columns are the
mixers' projections side by side, and the heads that each mixer leaves (already times its constant, in 32-bit before
they are rounded) lie side by side in one row for the second, whose matrix is the output matrices side by side.  A mixer
that can stand here says how many columns it reads and leaves (`in_cols`, `out_cols`), has its two matrices as `w_in` and
`w_o`, its output bias (times its constant) as `out_bias`, and does what lies between as `run_heads`.  Each keeps the
cache and the state it would keep alone; one of them at most may keep keys and values.
"""
from __future__ import annotations

from typing import List, Mapping, Optional

import torch

from .. import ops
from ..errors import SpecError
from ..registry import part_impl, register_part
from . import linear
from .base import CallStore, KVNeed, Mixer, StateNeed, StepInfo, WeightSpec


class ParallelMixers(Mixer):
    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        specs = spec.params["mixers"]                 # {name: PartSpec}; the name prefixes its state's names
        self.names = list(specs)
        self.mixers = [part_impl("mixer", s.kind)(s, rt) for s in specs.values()]
        for name, m in zip(self.names, self.mixers):
            if not hasattr(m, "run_heads"):
                raise SpecError(f"arch spec error: the mixer {name!r} cannot stand beside another one")
        if sum(m.kv_need() is not None for m in self.mixers) > 1:
            raise SpecError("arch spec error: one of the mixers side by side at most may keep keys and values")
        self.graph_safe = all(m.graph_safe for m in self.mixers)
        self.out_bias: Optional[torch.Tensor] = None
        self._stores = {}

    def weight_specs(self) -> List[WeightSpec]:
        return [s for m in self.mixers for s in m.weight_specs()]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for m in self.mixers:
            m.bind(tensors)

        def joined(mats, dim):
            if len({t.dtype for t in mats}) > 1:
                mats = [t.float() for t in mats]
            return torch.cat(mats, dim=dim).contiguous()
        self.w_in = linear.pad_rows(joined([m.w_in for m in self.mixers], 0))
        self.w_o = joined([m.w_o for m in self.mixers], 1)
        for m in self.mixers:
            m.w_in = m.w_o = None                     # held once, here
        biases = [m.out_bias for m in self.mixers if m.out_bias is not None]
        self.out_bias = torch.stack(biases).sum(0).contiguous() if biases else None

    def kv_need(self) -> Optional[KVNeed]:
        return next((m.kv_need() for m in self.mixers if m.kv_need() is not None), None)

    def state_needs(self) -> List[StateNeed]:
        return [StateNeed(f"{name}.{s.name}", s.shape, s.dtype)
                for name, m in zip(self.names, self.mixers) for s in m.state_needs()]

    def _views(self, store: CallStore):
        """The store as each mixer sees it (made once per entry of the run order)."""
        kept = self._stores.get(id(store))
        if kept is None or kept[0] is not store:
            views = [CallStore(store.kv if m.kv_need() is not None else None, store.owns_kv,
                               {s.name: store.state[f"{name}.{s.name}"] for s in m.state_needs()})
                     for name, m in zip(self.names, self.mixers)]
            kept = self._stores[id(store)] = (store, views)
        return kept[1]

    def forward(self, h, step: StepInfo, store: CallStore):
        y = self._heads(h, step, store)
        if self.out_bias is not None:
            return linear.matmul(y, self.w_o, epilogue=ops.EPI_BIAS, bias=self.out_bias)
        return linear.matmul(y, self.w_o)

    def forward_unbiased(self, h, step: StepInfo, store: CallStore):
        """As forward, without `out_bias`, for a consumer that adds it; may hand back 32-bit partial sums."""
        return linear.matmul_or_partials(self._heads(h, step, store), self.w_o)

    def _heads(self, h, step, store):
        proj = linear.matmul(h, self.w_in, out_dtype=torch.float32)
        y = torch.empty((h.shape[0], self.w_o.shape[1]), dtype=h.dtype, device=h.device)
        col = out_col = 0
        for m, view in zip(self.mixers, self._views(store)):
            m.run_heads(proj, col, step, view, y, out_col)
            col, out_col = col + m.in_cols, out_col + m.out_cols
        return y


register_part("mixer", "parallel_mixers", ParallelMixers)
