"""Typed configuration of Nuvivik: a decoder-only model whose layers are listed one by one in config.json.  The branches
read the residual stream itself and only their outputs are normed.  The mixer is attention over a latent cache whose
queries go through a latent of their own (with a window, a sink and rotate-half pairs), or grouped-query softmax attention
(biases, rotated and then normalised queries and keys, scaled frequencies, a soft-cap and a window); the feed-forward is
dense, or experts chosen from the best groups, or absent.

    {"architecture": "Nuvivik", "vocab": V, "width": D, "norm": {"eps": e}, "embedding": {"scale": s},
     "logit_scale": m, "logit_softcap": c,
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads": H, "dim": d, "rot_dim": r, "vdim": v, "q_rank": Q, "kv_rank": R, "scale": s,
                           "mask": {"size": W}, "rot": {"base": b, "dims": r}}, "mlp": MLP or null},
                {"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": v, "scale": s, "softcap": c,
                           "mask": {"size": W},
                           "rot": {"base": b, "dims": n,
                                   "scaling": {"factor": f, "low": l, "high": h, "original": o}}}, ...}]}
    MLP = {"kind": "dense", "ff": F}
        | {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k, "groups": {"count": g, "keep": n}}}

`mask`, `rot.scaling`, `softcap`, `groups`, `logit_scale`, `logit_softcap`, `embedding.scale` and `mlp` may be absent (every
earlier key in sight, plain frequencies, plain scores, every expert open, factors of one, plain logits, no feed-forward).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Tuple

from ..errors import MissingMetaError
from .base import ConfigReader, ModelConfig

MIXER_TYPES = ("latent_attention", "attention")
MLP_KINDS = ("dense", "moe")
SCALING_KEYS = ("factor", "low", "high", "original")


def _section(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise MissingMetaError(f"missing model metadata: {where}{key} (an object is required)")
    return v


def _bad(msg: str):
    raise MissingMetaError("model metadata invalid: " + msg)


def _positive(r: ConfigReader, keys, where: str) -> None:
    for key in keys:
        if r.need_int(key) <= 0:
            _bad(f"{where}{key} must be positive")


def _rot(m: Mapping[str, Any], where: str, at_most: int) -> None:
    rot = _section(m, "rot", where)
    r = ConfigReader(rot)
    dims, base = r.need_int("dims"), r.opt_float("base", None)
    if base is None or not base > 0.0:
        _bad(f"{where}rot.base must be a positive number")
    if dims <= 0 or dims % 2 or dims > at_most:
        _bad(f"{where}rot.dims must be even and lie between 2 and {at_most}")
    if rot.get("scaling") is not None:
        sc = ConfigReader(_section(rot, "scaling", where + "rot."))
        for key in SCALING_KEYS:
            v = sc.opt_float(key, None)
            if v is None or not v > 0.0:
                _bad(f"{where}rot.scaling.{key} must be a positive number")
        if sc.opt_float("high", None) < sc.opt_float("low", None):
            _bad(f"{where}rot.scaling.high must not lie below rot.scaling.low")


def _mask(m: Mapping[str, Any], where: str) -> None:
    if m.get("mask") is not None and ConfigReader(_section(m, "mask", where)).need_int("size") <= 0:
        _bad(f"{where}mask.size must be positive")


@dataclass(frozen=True)
class NuvivikConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    logit_softcap: float                       # 0: plain logits
    layers: Tuple[Mapping[str, Any], ...]      # the entries as config.json has them, checked

    architecture = "Nuvivik"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "NuvivikConfig":
        r = ConfigReader(raw)
        eps = ConfigReader(_section(raw, "norm", "")).opt_float("eps", None)
        if eps is None:
            raise MissingMetaError("missing model metadata: norm.eps")
        emb = raw.get("embedding") if isinstance(raw.get("embedding"), dict) else {}
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise MissingMetaError("missing model metadata: layers (a list of layers is required)")
        cfg = cls(vocab=r.need_int("vocab"), width=r.need_int("width"), norm_eps=eps,
                  embedding_scale=ConfigReader(emb).opt_float("scale", 1.0), logit_scale=r.opt_float("logit_scale", 1.0),
                  logit_softcap=r.opt_float("logit_softcap", 0.0), layers=tuple(copy.deepcopy(l) for l in layers))
        cfg.check()
        return cfg

    def check(self) -> None:
        for key in ("vocab", "width"):
            if getattr(self, key) <= 0:
                _bad(f"{key} must be positive")
        if not self.norm_eps > 0.0:
            _bad("norm.eps must be positive")
        if self.logit_softcap < 0.0:
            _bad("logit_softcap cannot be negative")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            if not isinstance(layer, dict):
                _bad(f"layers[{i}] must be an object")
            kind = layer.get("type")
            if kind not in MIXER_TYPES:
                _bad(f"{where}type must be one of {MIXER_TYPES}, found {kind!r}")
            m = _section(layer, "mixer", where)
            getattr(self, "_check_" + kind)(m, where + "mixer.")
            self._check_mlp(layer.get("mlp"), where)

    @staticmethod
    def _check_latent_attention(m, where: str) -> None:
        r = ConfigReader(m)
        _positive(r, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"), where)
        if r.opt_float("scale", None) is None:
            _bad(f"{where}scale is required")
        _rot(m, where, r.need_int("rot_dim"))
        _mask(m, where)

    @staticmethod
    def _check_attention(m, where: str) -> None:
        r = ConfigReader(m)
        _positive(r, ("heads", "kv_heads", "dim", "vdim"), where)
        if r.need_int("heads") % r.need_int("kv_heads") != 0:
            _bad(f"{where}heads must be a multiple of {where}kv_heads")
        if r.opt_float("scale", None) is None:
            _bad(f"{where}scale is required")
        if r.opt_float("softcap", 0.0) < 0.0:
            _bad(f"{where}softcap cannot be negative")
        _rot(m, where, r.need_int("dim"))
        _mask(m, where)

    @staticmethod
    def _check_mlp(mlp, where: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") not in MLP_KINDS:
            _bad(f"{where}mlp.kind must be one of {MLP_KINDS} (or mlp null)")
        if mlp["kind"] == "dense":
            if ConfigReader(mlp).need_int("ff") <= 0:
                _bad(f"{where}mlp.ff must be positive")
            return
        router = ConfigReader(_section(mlp, "router", where + "mlp."))
        if ConfigReader(_section(mlp, "expert", where + "mlp.")).need_int("ff") <= 0:
            _bad(f"{where}mlp.expert.ff must be positive")
        n, top = router.need_int("experts"), router.need_int("top")
        if not 0 < top <= n:
            _bad(f"{where}mlp.router.top must lie between 1 and mlp.router.experts")
        if router.raw.get("groups") is not None:
            g = ConfigReader(_section(router.raw, "groups", where + "mlp.router."))
            count, keep = g.need_int("count"), g.need_int("keep")
            if count <= 0 or n % count != 0:
                _bad(f"{where}mlp.router.groups.count must divide mlp.router.experts")
            if not 0 < keep <= count:
                _bad(f"{where}mlp.router.groups.keep must lie between 1 and groups.count")
            if top > keep * (n // count):
                _bad(f"{where}mlp.router.top is more than the kept groups hold")

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
                "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap,
                "layers": [copy.deepcopy(dict(l)) for l in self.layers]}
