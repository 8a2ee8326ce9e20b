"""Nuvivik as data: the function from a `NuvivikConfig` to a `ModelPlan`.

Embedding: the token table times a constant.  Every layer is the branch-norm arrangement with plain RMS norms,
x += norm1(mixer(x)); x += norm2(ff(x)).  Mixers: attention over a latent cache with a latent for the queries, rotate-half
pairs, a window and a sink; grouped-query attention with biases, rotate-half pairs at banded frequencies on a part of
every head, queries and keys over their root mean square, a soft-cap and a window.  Feed-forward: down(gelu(up h)) in the
tanh form, or experts down(relu(up h)^2) with logistic scores, chosen from the best groups and weighted with their scores
as they are.  A last norm (the logits' factor folded into it), an untied head with a soft-cap.  Tensor names: `embed`,
`l<i>.norm1|norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.base import LayerCall, LayerSpec, ModelPlan, PartSpec
from ..config.nuvivik import SCALING_KEYS, NuvivikConfig
from ..registry import register_architecture

MAX_POSITIONS = 1 << 20        # the format names no limit: the cache alone bounds a sequence


def _rotary(rot) -> PartSpec:
    sc = rot.get("scaling")
    scaling = dict({k: float(sc[k]) for k in SCALING_KEYS}, kind="bands") if sc else None
    return PartSpec("rotary", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"]), "style": "rotate_half",
                               "table": "float64", "scaling": scaling})


def _mixer(cfg: NuvivikConfig, layer, p: str) -> PartSpec:
    m = layer["mixer"]
    window = int(m["mask"]["size"]) if m.get("mask") else None
    if layer["type"] == "latent_attention":
        return PartSpec("latent_attention",
                        {"width": cfg.width, "n_heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"],
                         "vdim": m["vdim"], "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "scale": float(m["scale"]),
                         "eps": cfg.norm_eps, "window": window, "sink": True, "position": _rotary(m["rot"])},
                        {"dq": p + "dq", "dq_norm": p + "dq.norm", "uq": p + "uq", "dkv": p + "dkv",
                         "dkv_norm": p + "dkv.norm", "uk": p + "uk", "uv": p + "uv", "sink": p + "sink", "o": p + "o"})
    return PartSpec("gated_softmax_attention",
                    {"width": cfg.width, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "dim": m["dim"],
                     "vdim": m["vdim"], "scale": float(m["scale"]), "eps": cfg.norm_eps, "window": window,
                     "softcap": float(m.get("softcap") or 0.0), "bias": True, "qk_norm": "unit",
                     "position": _rotary(m["rot"])},
                    {"q": p + "q", "k": p + "k", "v": p + "v", "q_bias": p + "q.b", "k_bias": p + "k.b",
                     "v_bias": p + "v.b", "o": p + "o"})


def _feed_forward(cfg: NuvivikConfig, layer, p: str) -> PartSpec:
    mlp = layer.get("mlp")
    if mlp is None:
        return PartSpec("none")
    if mlp["kind"] == "dense":
        return PartSpec("dense_mlp", {"width": cfg.width, "inner": mlp["ff"], "activation": "gelu_tanh", "bias": False},
                        {"up": p + "up", "down": p + "down"})
    router = mlp["router"]
    return PartSpec("routed_experts",
                    {"width": cfg.width, "inner": mlp["expert"]["ff"], "experts": router["experts"], "top": router["top"],
                     "identity": 0, "scoring": "logistic", "weight_on": "output", "correction": False,
                     "activation": "relu_square", "groups": dict(router["groups"]) if router.get("groups") else None},
                    {"router": p + "router", "expert": p + "e{}.", "up": "up", "down": "down"})


def nuvivik_plan(cfg: NuvivikConfig) -> ModelPlan:
    def norm(name: str, mult: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"width": cfg.width, "eps": cfg.norm_eps, "add_one": False, "mult": mult}, {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        norms = {"post_mixer": norm(p + "norm1")}
        if layer.get("mlp") is not None:
            norms["post_ffn"] = norm(p + "norm2")
        layers.append(LayerSpec("branch_norm", _mixer(cfg, layer, p + "mix."), _feed_forward(cfg, layer, p + "mlp."), norms))
    return ModelPlan(
        width=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=PartSpec("scaled_embedding", {"vocab": cfg.vocab, "width": cfg.width, "scale": cfg.embedding_scale},
                           {"table": "embed"}),
        layers=layers, schedule=[LayerCall(i) for i in range(len(layers))], final_norm=norm("final.norm", cfg.logit_scale),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "width": cfg.width, "softcap": cfg.logit_softcap}, {"table": "head"}),
    )


register_architecture("Nuvivik", NuvivikConfig, nuvivik_plan)
