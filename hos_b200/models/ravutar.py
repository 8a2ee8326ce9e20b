"""Ravutar as data: the function from a `RavutarConfig` to a `ModelPlan`.

Embedding: the token table, copied to every residual stream.  Every layer is the hyper-connections arrangement with plain
RMS norms before the mixer and the feed-forward.  Mixers: the state-space recurrence; or two mixers side by side, softmax
attention (biases on all four projections, a short convolution on every q, k and v channel, a query factor that grows with
the position, one added to the softmax's denominator, no rotation, every earlier key in sight) and linear attention with a
decay per key channel.  Feed-forward: dense with biases and the erf-form GELU.  The configuration's loop becomes repeated
calls of the same layers, each call with a cache and state of its own.  The factor on the logits is the last norm's `mult`.
Tensor names: `embed`, `l<i>.norm1|norm2`, `l<i>.hc1|hc2.in|out|mix`, `l<i>.mix.*` (side by side: `l<i>.mix.left.*`,
`l<i>.mix.right.*`), `l<i>.mlp.up|down` with `.b`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.base import LayerCall, LayerSpec, ModelPlan, PartSpec
from ..config.ravutar import RavutarConfig
from ..registry import register_architecture

MAX_POSITIONS = 1 << 20        # the format names no limit: the cache alone bounds a sequence


def _state_space(cfg: RavutarConfig, m, p: str) -> PartSpec:
    return PartSpec("state_space",
                    {"width": cfg.width, "n_heads": m["heads"], "vdim": m["vdim"], "state": m["state"], "groups": m["groups"],
                     "taps": m["conv"], "norm_groups": m["norm_groups"], "eps": cfg.norm_eps},
                    {"in": p + "in", "conv": p + "conv", "conv_bias": p + "conv.b", "dt_bias": p + "dt_bias", "A_log": p + "A_log",
                     "D": p + "D", "norm": p + "norm", "o": p + "o"})


def _side_by_side(cfg: RavutarConfig, m, p: str) -> PartSpec:
    left, right = m["left"], m["right"]
    lp, rp = p + "left.", p + "right."
    names = {"o": lp + "o", "o_bias": lp + "o.b"}
    for r in ("q", "k", "v"):
        names.update({r: lp + r, r + "_bias": lp + r + ".b", r + "_conv": lp + r + ".conv"})
    attention = PartSpec("gated_softmax_attention",
                         {"width": cfg.width, "n_heads": left["heads"], "n_kv_heads": left["kv_heads"], "dim": left["dim"],
                          "vdim": left["vdim"], "scale": float(left["scale"]), "bias": True, "o_bias": True, "sink": "zero",
                          "conv": left.get("conv"), "q_temp": left.get("q_temp"), "out_scale": float(m.get("left_scale", 1.0))},
                         names)
    linear = PartSpec("channel_decay_attention",
                      {"width": cfg.width, "n_heads": right["heads"], "dim": right["dim"], "vdim": right["vdim"],
                       "tau": float(right["tau"]), "decay_rank": right.get("decay_rank"), "eps": cfg.norm_eps,
                       "out_scale": float(m.get("right_scale", 1.0))},
                      {"q": rp + "q", "k": rp + "k", "v": rp + "v", "gate": rp + "g", "a1": rp + "a1", "a2": rp + "a2",
                       "a2_bias": rp + "a2.b", "norm": rp + "norm", "o": rp + "o"})
    return PartSpec("parallel_mixers", {"mixers": {"left": attention, "right": linear}})


def ravutar_plan(cfg: RavutarConfig) -> ModelPlan:
    def norm(name: str, mult: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"width": cfg.width, "eps": cfg.norm_eps, "add_one": False, "mult": mult}, {"weight": name})

    def mix(p: str):
        return {r: f"{p}.{r}" for r in ("in", "out", "mix")}

    layers = []
    for i, layer in enumerate(cfg.layers):
        p, mlp = f"l{i}.", layer.get("mlp")
        make = _state_space if layer["type"] == "mamba2" else _side_by_side
        norms, mixes = {"pre_mixer": norm(p + "norm1")}, {"mixer": mix(p + "hc1")}
        ff = PartSpec("none")
        if mlp is not None:
            norms["pre_ffn"], mixes["ffn"] = norm(p + "norm2"), mix(p + "hc2")
            ff = PartSpec("dense_mlp", {"width": cfg.width, "inner": mlp["ff"], "activation": "gelu_erf"},
                          {"up": p + "mlp.up", "up_bias": p + "mlp.up.b", "down": p + "mlp.down", "down_bias": p + "mlp.down.b"})
        layers.append(LayerSpec("hyper_prenorm", make(cfg, layer["mixer"], p + "mix."), ff, norms,
                                {"streams": cfg.streams, "mixes": mixes}))
    return ModelPlan(
        width=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=PartSpec("scaled_embedding", {"vocab": cfg.vocab, "width": cfg.width, "copies": cfg.streams}, {"table": "embed"}),
        layers=layers, schedule=[LayerCall(i) for i in cfg.run_order()], final_norm=norm("final.norm", cfg.logit_scale),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "width": cfg.width, "softcap": 0.0}, {"table": "head"}),
        streams=cfg.streams)


register_architecture("Ravutar", RavutarConfig, ravutar_plan)
