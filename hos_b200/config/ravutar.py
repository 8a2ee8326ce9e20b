"""Typed configuration of Ravutar: a decoder-only model whose layers are listed one by one in config.json and whose
residual stream is several copies of the width (hyper-connections).  The mixer is a state-space recurrence (Mamba-2's), or
softmax attention and a linear attention with a decay per key channel side by side; the feed-forward is a dense one with
biases, or absent.  A run of layers may be repeated with the same weights.

    {"architecture": "Ravutar", "vocab": V, "width": D, "streams": S, "norm": {"eps": e}, "logit_scale": m,
     "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "mamba2",
                 "mixer": {"heads": H, "vdim": v, "state": N, "groups": G, "conv": t, "norm_groups": P}, "mlp": MLP or null},
                {"type": "parallel",
                 "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": v, "scale": s, "conv": t,
                                    "q_temp": {"coef": c, "every": n}},
                           "right": {"heads": H, "dim": d, "vdim": v, "tau": x, "decay_rank": r},
                           "left_scale": l, "right_scale": r}, ...}]}
    MLP = {"kind": "dense", "ff": F}

`loop`, `logit_scale` (1), `left.q_temp`, `left.conv` (no convolution), `left_scale` and `right_scale` (1) and `mlp` may be absent;
`decay_rank` is needed for random weights only (a checkpoint's tensor gives it).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from ..errors import MissingMetaError
from .base import ConfigReader, ModelConfig

MIXER_TYPES = ("mamba2", "parallel")
MLP_KINDS = ("dense",)


def _section(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise MissingMetaError(f"missing model metadata: {where}{key} (an object is required)")
    return v


def _bad(msg: str):
    raise MissingMetaError("model metadata invalid: " + msg)


def _positive(r: ConfigReader, keys, where: str) -> None:
    for key in keys:
        try:
            v = r.need_int(key)
        except MissingMetaError as e:
            raise MissingMetaError(f"{e} in {where}") from None
        if v <= 0:
            _bad(f"{where}{key} must be positive")


@dataclass(frozen=True)
class RavutarConfig(ModelConfig):
    vocab: int
    width: int
    streams: int
    norm_eps: float
    logit_scale: float
    loop: Optional[Mapping[str, int]]
    layers: Tuple[Mapping[str, Any], ...]      # the entries as config.json has them, checked

    architecture = "Ravutar"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "RavutarConfig":
        r = ConfigReader(raw)
        eps = ConfigReader(_section(raw, "norm", "")).opt_float("eps", None)
        if eps is None:
            raise MissingMetaError("missing model metadata: norm.eps")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise MissingMetaError("missing model metadata: layers (a list of layers is required)")
        loop = None
        if raw.get("loop") is not None:
            lr = ConfigReader(_section(raw, "loop", ""))
            loop = {k: lr.need_int(k) for k in ("start", "stop", "times")}
        cfg = cls(vocab=r.need_int("vocab"), width=r.need_int("width"), streams=r.need_int("streams"), norm_eps=eps,
                  logit_scale=r.opt_float("logit_scale", 1.0), loop=loop, layers=tuple(copy.deepcopy(l) for l in layers))
        cfg.check()
        return cfg

    def check(self) -> None:
        for key in ("vocab", "width", "streams"):
            if getattr(self, key) <= 0:
                _bad(f"{key} must be positive")
        if not self.norm_eps > 0.0:
            _bad("norm.eps must be positive")
        if self.loop is not None and not (0 <= self.loop["start"] < self.loop["stop"] <= len(self.layers) and self.loop["times"] >= 1):
            _bad("loop.start, loop.stop and loop.times must name a run of layers and how often it runs")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            if not isinstance(layer, dict):
                _bad(f"layers[{i}] must be an object")
            kind = layer.get("type")
            if kind not in MIXER_TYPES:
                _bad(f"{where}type must be one of {MIXER_TYPES}, found {kind!r}")
            getattr(self, "_check_" + kind)(_section(layer, "mixer", where), where + "mixer.")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") not in MLP_KINDS:
                _bad(f"{where}mlp.kind must be one of {MLP_KINDS} (or mlp null)")
            _positive(ConfigReader(mlp), ("ff",), where + "mlp.")

    @staticmethod
    def _check_mamba2(m, where: str) -> None:
        r = ConfigReader(m)
        _positive(r, ("heads", "vdim", "state", "groups", "conv", "norm_groups"), where)
        if m["heads"] % m["groups"] != 0:
            _bad(f"{where}heads must be a multiple of {where}groups")
        if m["heads"] * m["vdim"] % m["norm_groups"] != 0:
            _bad(f"{where}norm_groups must divide heads x vdim")

    @staticmethod
    def _check_parallel(m, where: str) -> None:
        left, right = _section(m, "left", where), _section(m, "right", where)
        r = ConfigReader(left)
        _positive(r, ("heads", "kv_heads", "dim", "vdim"), where + "left.")
        if left["heads"] % left["kv_heads"] != 0:
            _bad(f"{where}left.heads must be a multiple of {where}left.kv_heads")
        if r.opt_float("scale", None) is None:
            _bad(f"{where}left.scale is required")
        if left.get("conv") is not None:
            _positive(r, ("conv",), where + "left.")
        if left.get("q_temp") is not None:
            t = ConfigReader(_section(left, "q_temp", where + "left."))
            if t.opt_float("coef", None) is None:
                _bad(f"{where}left.q_temp.coef is required")
            _positive(t, ("every",), where + "left.q_temp.")
        r = ConfigReader(right)
        _positive(r, ("heads", "dim", "vdim"), where + "right.")
        tau = r.opt_float("tau", None)
        if tau is None or not tau > 0.0:
            _bad(f"{where}right.tau must be a positive number")
        if right.get("decay_rank") is not None:
            _positive(r, ("decay_rank",), where + "right.")
        for key in ("left_scale", "right_scale"):
            ConfigReader(m).opt_float(key, 1.0)

    def run_order(self) -> List[int]:
        """The layers in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b = self.loop["start"], self.loop["stop"]
        return list(range(a)) + list(range(a, b)) * self.loop["times"] + list(range(b, n))

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
               "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale,
               "layers": [copy.deepcopy(dict(l)) for l in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        return out
