"""Shared by the Ravutar tests: small configurations that differ from one another in every size and constant, model
folders with random weights scaled so that every mechanism matters to the logits (sharp attention, decays that remember
far back, step sizes around one, mixing weights that neither vanish nor explode), and the comparison rules.

Tolerances, fixed before the first run (the ones the other designs' tests use): 32-bit: every row's error (root mean
square over the vocabulary) at most 2e-5 of the logits' root mean square; bfloat16: at most 4e-2 of it for at least
nine rows in ten."""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Optional

import torch

from satapel_cases import assert_rows, oracle_view, row_errors, tokens  # noqa: F401  (the rules are the same)


def mamba2(heads, vdim, state, groups, conv, norm_groups, mlp="dense"):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                                   "norm_groups": norm_groups}}


def left(heads, kv_heads, dim, vdim, scale, conv, q_temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if q_temp:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return m


def right(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}


def parallel(l, r, scales=(1.0, 1.0), mlp="dense"):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": l, "right": r, "left_scale": scales[0], "right_scale": scales[1]}}


def model(width, vocab, layers, streams, ff=48, eps=1e-6, logit_scale=1.0, loop=None):
    out = []
    for layer in layers:
        layer = json.loads(json.dumps(layer))
        if layer["mlp"] == "dense":
            layer["mlp"] = {"kind": "dense", "ff": ff}
        out.append(layer)
    raw = {"architecture": "Ravutar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
           "logit_scale": logit_scale, "layers": out}
    if loop:
        raw["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return raw


# side by side first, inside a loop with a state-space layer; three query heads to a kv head, keys wider than values, a
# query factor that steps every 16 positions; norm groups that cut through heads; a layer without a feed-forward
CASE_A = model(72, 211, [parallel(left(3, 1, 24, 16, 0.6, 4, (0.4, 16)), right(2, 12, 20, 8.0, 5), (0.7, 1.1)),
                         mamba2(6, 12, 20, 3, 3, 4),
                         parallel(left(2, 2, 8, 24, 0.9, 2, (1.5, 7)), right(3, 8, 8, 2.0, 9), (1.3, 0.5), mlp=None)],
               streams=3, ff=56, logit_scale=0.6, loop=(0, 2, 2))
# no loop, no query factor; one group and one norm part; two streams; a tau of one; values wider than a head of keys
CASE_B = model(64, 150, [mamba2(2, 40, 8, 1, 2, 1, mlp=None),
                         parallel(left(4, 4, 16, 40, 0.4, 3), right(1, 32, 8, 1.0, 16)),
                         mamba2(8, 8, 16, 8, 4, 8)], streams=2, ff=40, eps=1e-5, logit_scale=3.0)
# one stream; convolutions of one tap; a query factor that steps at every position; the loop at the end, three times
CASE_C = model(80, 90, [mamba2(4, 16, 12, 2, 1, 2),
                        parallel(left(8, 2, 8, 8, 0.7, 1, (0.3, 1)), right(4, 16, 12, 32.0, 3), (0.9, 0.8))],
               streams=1, ff=24, loop=(1, 2, 3))
# sizes that are multiples of nothing (a width of 100: the tensor-core products step aside), five streams, five taps
CASE_D = model(100, 77, [parallel(left(5, 5, 6, 10, 0.8, 5, (0.8, 33)), right(3, 10, 6, 5.0, 7), (0.5, 1.4)),
                         mamba2(5, 6, 30, 5, 6, 3),
                         parallel(left(6, 2, 10, 6, 0.7, 2, (0.2, 3)), right(2, 6, 18, 12.0, 1), mlp=None)],
               streams=5, ff=36, eps=3e-5, logit_scale=1.5, loop=(1, 3, 2))
# wider layers: heads of 64 and 128 numbers (the tensor-core attention kernels), states of 64 x 128 and 128 x 64, inner
# sizes of several hundred, a feed-forward of several tiles
CASE_E = model(320, 500, [parallel(left(8, 2, 64, 128, 0.15, 4, (0.3, 100)), right(4, 64, 96, 16.0, 24), (0.8, 1.2)),
                          mamba2(8, 64, 128, 2, 4, 4),
                          parallel(left(4, 4, 128, 64, 0.1, 3), right(2, 128, 128, 8.0, 8), (1.1, 0.6), mlp=None)],
               streams=4, ff=520, logit_scale=2.5, loop=(0, 2, 2))
# seeds for which 32-bit rounding alone (the oracle in 32-bit against itself) stays below 4e-6 of the logits' size: a head norm
# of a read-out that happens to be near zero amplifies whatever it is given
CASES = {"A": (CASE_A, 70), "B": (CASE_B, 65), "C": (CASE_C, 54), "D": (CASE_D, 58), "E": (CASE_E, 59)}


def _scaled(name: str, t: torch.Tensor) -> torch.Tensor:
    t = t.float()
    if name.endswith(("norm1", "norm2", "final.norm", "mix.norm", "right.norm")):
        return 1.0 + t
    if name.endswith(("hc1.mix", "hc2.mix")):          # near a permutation-free mix: the streams neither vanish nor explode
        return 0.8 * torch.eye(t.shape[0]) + 0.4 * t / t.shape[0] ** 0.5 * 2.0
    if name.endswith(("hc1.in", "hc2.in")):
        return 0.6 + 0.6 * t
    if name.endswith(("hc1.out", "hc2.out")):
        return 0.5 + 0.8 * t
    if name == "embed":
        return t * 50.0
    if name == "head":
        return t * 10.0
    if name.endswith(("left.q", "left.k")):
        return t * 6.0
    if name.endswith(("left.q.b", "left.k.b", "left.v.b", "left.o.b")):
        return t * 4.0
    if name.endswith(("left.q.conv", "left.k.conv", "left.v.conv")):
        t = t.clone()
        t[:, -1] += 0.7
        return t
    if name.endswith("mix.conv"):
        t = t.clone()
        t[:, -1] += 0.6
        return t
    if name.endswith(("left.v", "up", "down", "right.k", "right.v", "right.g", "right.q")):
        return t * 3.0
    if name.endswith(("up.b", "down.b", "conv.b")):
        return t * 3.0
    if name.endswith("a2.b"):
        return 1.0 + 2.0 * t
    if name.endswith("a2"):
        return t * 4.0
    if name.endswith("A_log"):
        return t - 2.0
    if name.endswith(("left.o", "right.o", "mix.o")):
        return t * 5.0
    return t


def make_folder(tmp_path, raw: dict, seed: int, name: str = "m",
                edit: Optional[Callable[[Dict[str, torch.Tensor]], None]] = None) -> str:
    from hos_b200.model import weight_specs_for
    from hos_b200.registry import config_from_dict
    from hos_b200.weights import RandomSource
    from hos_b200.weights.safetensors import SINGLE_FILE, write_safetensors
    cfg = config_from_dict(raw)
    src = RandomSource(weight_specs_for(cfg), seed)
    tensors = {n: _scaled(n, src.read(n)) for n in src.names()}
    if edit is not None:
        edit(tensors)
    d = os.path.join(str(tmp_path), name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg.to_dict(), f)
    write_safetensors(os.path.join(d, SINGLE_FILE), ((n, t.to(torch.bfloat16)) for n, t in tensors.items()),
                      metadata={"format": "pt"})
    return d
