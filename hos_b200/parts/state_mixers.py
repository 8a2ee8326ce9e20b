"""Mixers that keep a matrix state S [dim keys x vdim values] per head and sequence instead of keys and values.

decay_linear_attention: q, k = act(W_q h), act(W_k h) (heads x dim), v = act(W_v h) (heads x vdim), act(x) = x
    logistic(x); per head S <- decay_h S + k v^T, o = S^T q with a constant decay per head and no other scale; the
    heads' outputs, side by side, are divided by their common root mean square, multiplied by a weight per column
    and by logistic(W_g h), and projected by W_o.  Each piece is a parameter: `activation` ("x_logistic", or None for
    q, k, v as projected); `position` (a rotary part: q and k turn with the token's position after the activation,
    angles in 32-bit); `key_scale` (a constant on k after the rotation); `norm` ("row": one root mean square over all
    heads; "head": one per head) with or without a weight (`norm_weight`); `gate` ("logistic" or "x_logistic").
gated_delta_rule: q, k (kv_heads x dim) and v (heads x vdim) each pass a short causal convolution over time per
    channel (`taps` wide, zeros before a sequence's start) and x logistic(x); q and k are divided by their lengths
    (sqrt(sum + 1e-6)) per head, q also by sqrt(dim); beta = logistic(W_b h) and the decay
    g = exp(-exp(A_log) softplus(W_a h + dt_bias)) are one number per head and token.  Per head (value head h reads
    key head h // (heads / kv_heads)):  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.  Each head's o
    is divided by its root mean square, multiplied by a weight shared by the heads and by W_g h times its logistic
    function, and projected by W_o.

channel_decay_attention: q = W_q h, k = W_k h (heads x dim), v = W_v h (heads x vdim) as projected; a decay per key channel
    alpha = logistic(W_a2 (W_a1 h) + b)^(1 / tau).  Per head S <- diag(alpha) S + k v^T, o = dim^-1/2 S^T q; each head's o is
    divided by its root mean square, multiplied by a weight shared by the heads and by W_g h times its logistic
    function (`out_scale`: and by a constant), and projected by W_o.
state_space: one projection gives [z | x | B | C | dt] (x, z: heads x vdim; B, C: groups x state; dt: heads).  x, B and C
    pass a short causal convolution over time per channel with a bias, and x logistic(x); dt = softplus(dt + dt_bias).
    Per head (head h reads group h // (heads / groups)):  S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x.  The
    heads' y, side by side, are multiplied by z logistic(z), then divided by their root mean square in `norm_groups`
    equal parts and multiplied by a weight per column, and projected by W_o.

The state (and the convolution's last taps - 1 inputs) is per-sequence state of fixed size: zero at a sequence's
start, carried from step to step.  Everything between the projections and the output projection is 32-bit: the
projections are one product that writes 32-bit rows.
"""
from __future__ import annotations

from typing import List, Mapping

import torch

from .. import ops
from ..errors import SpecError
from ..registry import part_impl, register_part
from . import linear
from .base import CallStore, Mixer, StateNeed, StepInfo, WeightSpec


class DecayLinearAttention(Mixer):
    graph_safe = True

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = spec.params
        self.width, self.n_heads = int(p["width"]), int(p["n_heads"])
        self.dim, self.vdim, self.eps = int(p["dim"]), int(p["vdim"]), float(p["eps"])
        self.decay = [float(d) for d in p["decay"]]
        if min(self.width, self.n_heads, self.dim, self.vdim) <= 0 or len(self.decay) != self.n_heads:
            raise SpecError("arch spec error: the decay mixer needs positive sizes and one decay per head")
        self.qk_cols, self.v_cols = self.n_heads * self.dim, self.n_heads * self.vdim
        act, norm, gate = p.get("activation", "x_logistic"), p.get("norm", "row"), p.get("gate", "logistic")
        if act not in (None, "x_logistic") or norm not in ("row", "head") or gate not in ("logistic", "x_logistic"):
            raise SpecError(f"arch spec error: the decay mixer with activation {act!r}, norm {norm!r}, gate {gate!r}")
        self.activates, self.norm_per_head = act is not None, norm == "head"
        self.norm_weight = bool(p.get("norm_weight", True))
        self.gate_act = ops.ACT_X_LOGISTIC if gate == "x_logistic" else ops.ACT_LOGISTIC
        self.key_scale = float(p.get("key_scale", 1.0))
        pos_spec = p.get("position")
        self.position = part_impl("position", pos_spec.kind)(pos_spec, rt) if pos_spec else None

    def weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        out = [WeightSpec(w["q"], (self.qk_cols, self.width), "matrix", 0.05),
               WeightSpec(w["k"], (self.qk_cols, self.width), "matrix", 0.05),
               WeightSpec(w["v"], (self.v_cols, self.width), "matrix", 0.05),
               WeightSpec(w["gate"], (self.v_cols, self.width), "matrix", 0.05),
               WeightSpec(w["o"], (self.width, self.v_cols), "matrix", 0.02)]
        if self.norm_weight:       # a weight per column, or one shared by the heads where the norm is per head
            out.append(WeightSpec(w["norm"], (self.vdim if self.norm_per_head else self.v_cols,), "vector", 0.1))
        return out

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        w = self.spec.weights
        mats = [self._matrix(tensors[w[r]]) for r in ("q", "k", "v", "gate")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        self.w_in = torch.cat(mats, dim=0).contiguous()
        self.w_o = self._matrix(tensors[w["o"]])
        if self.norm_weight:
            self.norm_w = self._vector32(tensors[w["norm"]])
        else:
            self.norm_w = torch.ones(self.vdim if self.norm_per_head else self.v_cols, dtype=torch.float32,
                                     device=self.w_o.device)
        self.decay_t = torch.tensor(self.decay, dtype=torch.float64).to(torch.float32).to(self.w_o.device)

    def state_needs(self) -> List[StateNeed]:
        return [StateNeed("S", (self.n_heads, self.vdim, self.dim), torch.float32)]      # kept as S^T per head

    def forward(self, h, step: StepInfo, store: CallStore):
        return self._run(h, step, store, False)

    def forward_partial(self, h, step: StepInfo, store: CallStore):
        return self._run(h, step, store, True)

    def _run(self, h, step, store, partial_ok):
        n = h.shape[0]
        proj = linear.matmul(h, self.w_in, out_dtype=torch.float32)
        o = torch.empty((n, self.v_cols), dtype=torch.float32, device=h.device)
        turns = self.position is not None or self.key_scale != 1.0
        rot = None
        if turns:
            # the rotation follows the activation, so the activation cannot ride in the scan's walk here
            if self.activates:
                ops.act_rows(proj, 2 * self.qk_cols + self.v_cols)
            freq, rot_dims, style = self.position.kernel_args() if self.position else (None, 0, 0)
            if step.max_new == 1 and not self.activates:
                rot = (freq, rot_dims, style, self.key_scale)       # single tokens: the scan turns what it stages
            else:
                ops.rotate_rows(proj, self.n_heads, self.n_heads, self.dim, freq, rot_dims, style, step, self.key_scale)
        ops.state_scan(proj, 0, self.qk_cols, 2 * self.qk_cols, self.activates and not turns, self.decay_t, False, None,
                       store.state["S"], step, o, self.n_heads, self.n_heads, self.dim, self.vdim, rot=rot)
        y = torch.empty((n, self.v_cols), dtype=h.dtype, device=h.device)
        if self.norm_per_head:
            ops.group_norm_gate(o, self.norm_w, proj, 2 * self.qk_cols + self.v_cols, self.gate_act, step.token_seq, y,
                                self.eps, self.n_heads, self.vdim)
        else:
            ops.group_norm_gate(o, self.norm_w, proj, 2 * self.qk_cols + self.v_cols, self.gate_act, step.token_seq, y,
                                self.eps, 1, self.v_cols)
        return linear.matmul_or_partials(y, self.w_o) if partial_ok else linear.matmul(y, self.w_o)


class GatedDeltaRule(Mixer):
    graph_safe = True

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = spec.params
        self.width, self.n_heads, self.n_kv_heads = int(p["width"]), int(p["n_heads"]), int(p["n_kv_heads"])
        self.dim, self.vdim, self.taps, self.eps = int(p["dim"]), int(p["vdim"]), int(p["taps"]), float(p["eps"])
        if min(self.width, self.n_heads, self.n_kv_heads, self.dim, self.vdim, self.taps) <= 0 \
                or self.n_heads % self.n_kv_heads != 0:
            raise SpecError("arch spec error: the delta-rule mixer needs positive sizes and heads that are a multiple of "
                            "its key heads")
        self.qk_cols, self.v_cols = self.n_kv_heads * self.dim, self.n_heads * self.vdim
        self.conv_cols = 2 * self.qk_cols + self.v_cols

    def weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        out = []
        for r, rows in (("q", self.qk_cols), ("k", self.qk_cols), ("v", self.v_cols)):
            out.append(WeightSpec(w[r], (rows, self.width), "matrix", 0.05))
            out.append(WeightSpec(w[r + "_conv"], (rows, self.taps), "matrix", 0.4))
        out += [WeightSpec(w["beta"], (self.n_heads, self.width), "matrix", 0.05),
                WeightSpec(w["a"], (self.n_heads, self.width), "matrix", 0.05),
                WeightSpec(w["A_log"], (self.n_heads,), "vector", 0.5),
                WeightSpec(w["dt_bias"], (self.n_heads,), "vector", 0.5),
                WeightSpec(w["gate"], (self.v_cols, self.width), "matrix", 0.05),
                WeightSpec(w["norm"], (self.vdim,), "vector", 0.1),
                WeightSpec(w["o"], (self.width, self.v_cols), "matrix", 0.02)]
        return out

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        w = self.spec.weights
        mats = [self._matrix(tensors[w[r]]) for r in ("q", "k", "v", "beta", "a", "gate")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        self.w_in = torch.cat(mats, dim=0).contiguous()           # q | k | v | beta | a | gate
        self.conv_w = torch.cat([tensors[w[r + "_conv"]].to(torch.float32) for r in ("q", "k", "v")], dim=0).contiguous()
        self.a_log, self.dt_bias = self._vector32(tensors[w["A_log"]]), self._vector32(tensors[w["dt_bias"]])
        self.norm_w = self._vector32(tensors[w["norm"]])
        self.w_o = self._matrix(tensors[w["o"]])

    def state_needs(self) -> List[StateNeed]:
        return [StateNeed("S", (self.n_heads, self.vdim, self.dim), torch.float32),
                StateNeed("conv", (max(self.taps - 1, 0), self.conv_cols), torch.float32)]

    def forward(self, h, step: StepInfo, store: CallStore):
        return self._run(h, step, store, False)

    def forward_partial(self, h, step: StepInfo, store: CallStore):
        return self._run(h, step, store, True)

    def _run(self, h, step, store, partial_ok):
        n, dev = h.shape[0], h.device
        raw = linear.matmul(h, self.w_in, out_dtype=torch.float32)
        act = torch.empty((n, self.conv_cols), dtype=torch.float32, device=dev)
        beta = torch.empty((n, self.n_heads), dtype=torch.float32, device=dev)
        g = torch.empty((n, self.n_heads), dtype=torch.float32, device=dev)
        kept = store.state["conv"]
        single = step.max_new == 1           # every sequence brings one token: the kept inputs move on in conv_prep itself
        ops.conv_prep(raw, self.conv_w, kept, self.a_log, self.dt_bias, step, act, beta, g, self.n_heads, self.n_kv_heads,
                      self.dim, self.vdim, keep_here=single)
        if not single:
            ops.conv_keep(raw, self.taps, kept, step, self.conv_cols)
        o = torch.empty((n, self.v_cols), dtype=torch.float32, device=dev)
        ops.state_scan(act, 0, self.qk_cols, 2 * self.qk_cols, False, g, True, beta, store.state["S"], step, o,
                       self.n_heads, self.n_kv_heads, self.dim, self.vdim)
        y = torch.empty((n, self.v_cols), dtype=h.dtype, device=dev)
        ops.group_norm_gate(o, self.norm_w, raw, self.conv_cols + 2 * self.n_heads, ops.ACT_X_LOGISTIC, step.token_seq, y,
                            self.eps, self.n_heads, self.vdim)
        return linear.matmul_or_partials(y, self.w_o) if partial_ok else linear.matmul(y, self.w_o)


class ChannelDecayAttention(Mixer):
    graph_safe = True
    out_bias = None

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = spec.params
        self.width, self.n_heads = int(p["width"]), int(p["n_heads"])
        self.dim, self.vdim, self.eps, self.tau = int(p["dim"]), int(p["vdim"]), float(p["eps"]), float(p["tau"])
        self.rank = int(p["decay_rank"]) if p.get("decay_rank") else -1          # -1: the a1 tensor's shape gives it
        self.out_scale = float(p.get("out_scale", 1.0))
        if min(self.width, self.n_heads, self.dim, self.vdim) <= 0 or not self.tau > 0.0:
            raise SpecError("arch spec error: the mixer with a decay per key channel needs positive sizes and a positive tau")
        self.qk_cols, self.v_cols = self.n_heads * self.dim, self.n_heads * self.vdim

    def weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        return [WeightSpec(w["q"], (self.qk_cols, self.width), "matrix", 0.05),
                WeightSpec(w["k"], (self.qk_cols, self.width), "matrix", 0.05),
                WeightSpec(w["v"], (self.v_cols, self.width), "matrix", 0.05),
                WeightSpec(w["gate"], (self.v_cols, self.width), "matrix", 0.05),
                WeightSpec(w["a1"], (self.rank, self.width), "matrix", 0.05),
                WeightSpec(w["a2"], (self.qk_cols, self.rank), "matrix", 0.1),
                WeightSpec(w["a2_bias"], (self.qk_cols,), "vector", 0.5),
                WeightSpec(w["norm"], (self.vdim,), "vector", 0.1),
                WeightSpec(w["o"], (self.width, self.v_cols), "matrix", 0.02)]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        w = self.spec.weights
        mats = [self._matrix(tensors[w[r]]) for r in ("q", "k", "v", "gate", "a1")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        self.bound_rank = mats[-1].shape[0]
        if tensors[w["a2"]].shape[1] != self.bound_rank:
            raise SpecError(f"arch spec error: the decay's two projections do not fit ({tuple(mats[-1].shape)}, "
                            f"{tuple(tensors[w['a2']].shape)})")
        self.w_in = torch.cat(mats, dim=0).contiguous()                          # q | k | v | gate | low-rank decay
        self.a2_t = tensors[w["a2"]].to(torch.float32).t().contiguous()          # [rank, heads * dim]
        self.a2_bias = self._vector32(tensors[w["a2_bias"]])
        self.norm_w = (self._vector32(tensors[w["norm"]]) * self.out_scale).contiguous()
        self.w_o = self._matrix(tensors[w["o"]])

    def state_needs(self) -> List[StateNeed]:
        return [StateNeed("S", (self.n_heads, self.vdim, self.dim), torch.float32)]      # kept as S^T per head

    def forward(self, h, step: StepInfo, store: CallStore):
        return linear.matmul(self._heads(h, step, store), self.w_o)

    def forward_partial(self, h, step: StepInfo, store: CallStore):
        return linear.matmul_or_partials(self._heads(h, step, store), self.w_o)

    def _heads(self, h, step, store):
        proj = linear.matmul(h, self.w_in, out_dtype=torch.float32)
        y = torch.empty((h.shape[0], self.v_cols), dtype=h.dtype, device=h.device)
        self.run_heads(proj, 0, step, store, y, 0)
        return y

    # the mixer between its projections (see parts/parallel_mixers.py)
    @property
    def in_cols(self) -> int:
        return 2 * self.qk_cols + 2 * self.v_cols + self.bound_rank

    @property
    def out_cols(self) -> int:
        return self.v_cols

    def run_heads(self, proj, col: int, step: StepInfo, store: CallStore, y, out_col: int) -> None:
        """From the projections (32-bit rows, columns from `col` on) to the gated heads in y's columns from out_col on."""
        n, dev = proj.shape[0], proj.device
        gate_col = col + 2 * self.qk_cols + self.v_cols
        alpha = torch.empty((n, self.qk_cols), dtype=torch.float32, device=dev)
        ops.channel_decay(proj, gate_col + self.v_cols, self.bound_rank, self.a2_t, self.a2_bias, self.tau, alpha)
        o = torch.empty((n, self.v_cols), dtype=torch.float32, device=dev)
        ops.state_scan(proj, col, col + self.qk_cols, col + 2 * self.qk_cols, False, alpha, True, None, store.state["S"], step, o,
                       self.n_heads, self.n_heads, self.dim, self.vdim, channel_g=True, o_mult=float(self.dim) ** -0.5)
        ops.group_norm_gate(o, self.norm_w, proj, gate_col, ops.ACT_X_LOGISTIC, step.token_seq, y, self.eps, self.n_heads, self.vdim,
                            out_col)


class StateSpace(Mixer):
    graph_safe = True

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        p = spec.params
        self.width, self.n_heads, self.vdim = int(p["width"]), int(p["n_heads"]), int(p["vdim"])
        self.state, self.groups, self.taps = int(p["state"]), int(p["groups"]), int(p["taps"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p["eps"])
        if min(self.width, self.n_heads, self.vdim, self.state, self.groups, self.taps, self.norm_groups) <= 0 \
                or self.n_heads % self.groups != 0 or (self.n_heads * self.vdim) % self.norm_groups != 0:
            raise SpecError("arch spec error: the state-space mixer needs positive sizes, heads that are a multiple of its groups "
                            "and an inner size that is a multiple of its norm groups")
        self.inner, self.bc_cols = self.n_heads * self.vdim, self.groups * self.state
        self.conv_cols = self.inner + 2 * self.bc_cols
        self.rows = self.inner + self.conv_cols + self.n_heads

    def weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        return [WeightSpec(w["in"], (self.rows, self.width), "matrix", 0.05),
                WeightSpec(w["conv"], (self.conv_cols, self.taps), "matrix", 0.4),
                WeightSpec(w["conv_bias"], (self.conv_cols,), "vector", 0.1),
                WeightSpec(w["dt_bias"], (self.n_heads,), "vector", 0.5),
                WeightSpec(w["A_log"], (self.n_heads,), "vector", 0.5),
                WeightSpec(w["D"], (self.n_heads,), "vector", 0.5),
                WeightSpec(w["norm"], (self.inner,), "vector", 0.1),
                WeightSpec(w["o"], (self.width, self.inner), "matrix", 0.02)]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        w = self.spec.weights
        self.w_in = linear.pad_rows(self._matrix(tensors[w["in"]]))              # z | x | B | C | dt
        self.conv_w = tensors[w["conv"]].to(torch.float32).t().contiguous()      # [taps, channels]
        self.conv_bias = self._vector32(tensors[w["conv_bias"]])
        self.dt_bias, self.a_log, self.skip = (self._vector32(tensors[w[r]]) for r in ("dt_bias", "A_log", "D"))
        self.norm_w = self._vector32(tensors[w["norm"]])
        self.w_o = self._matrix(tensors[w["o"]])

    def state_needs(self) -> List[StateNeed]:
        out = [StateNeed("S", (self.n_heads, self.vdim, self.state), torch.float32)]     # kept as S^T per head
        if self.taps > 1:
            out.append(StateNeed("conv", (self.taps - 1, self.conv_cols), torch.float32))
        return out

    def forward(self, h, step: StepInfo, store: CallStore):
        return linear.matmul(self._heads(h, step, store), self.w_o)

    def forward_partial(self, h, step: StepInfo, store: CallStore):
        return linear.matmul_or_partials(self._heads(h, step, store), self.w_o)

    def _heads(self, h, step, store):
        n, dev = h.shape[0], h.device
        raw = linear.matmul(h, self.w_in, out_dtype=torch.float32)
        act = torch.empty((n, self.conv_cols), dtype=torch.float32, device=dev)
        dt = torch.empty((n, self.n_heads), dtype=torch.float32, device=dev)
        g = torch.empty_like(dt)
        kept = store.state["conv"] if self.taps > 1 else raw.new_empty((0, 0, self.conv_cols))
        single = step.max_new == 1           # every sequence brings one token: the kept inputs move on in the same launch
        ops.conv_act_rows(raw, self.inner, self.conv_w, self.conv_bias, kept, "x_logistic", step, act, single,
                          (self.inner + self.conv_cols, self.dt_bias, self.a_log, dt, g))
        if self.taps > 1 and not single:
            ops.conv_keep(raw, self.taps, kept, step, self.conv_cols, self.inner)
        o = torch.empty((n, self.inner), dtype=torch.float32, device=dev)
        ops.state_scan(act, self.inner + self.bc_cols, self.inner, 0, False, g, True, None, store.state["S"], step, o,
                       self.n_heads, self.groups, self.state, self.vdim, v_factor=dt)
        y = torch.empty((n, self.inner), dtype=h.dtype, device=dev)
        ops.skip_gate_norm(o, act, 0, self.skip, raw, 0, self.norm_w, self.eps, step.token_seq, y, self.n_heads, self.vdim,
                           self.norm_groups)
        return y


register_part("mixer", "channel_decay_attention", ChannelDecayAttention)
register_part("mixer", "state_space", StateSpace)
register_part("mixer", "decay_linear_attention", DecayLinearAttention)
register_part("mixer", "gated_delta_rule", GatedDeltaRule)
