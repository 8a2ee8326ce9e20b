"""Shared by the Nuvivik tests: small configurations that differ from one another in every size and constant, model
folders with random weights scaled so that every mechanism matters to the logits (sharp attention, a soft-cap that bites,
sinks of the size of the scores, router logits of a few units), and the comparison rules.

Tolerances, fixed before the first run (the ones the other designs' tests use): 32-bit: every row's error (root mean
square over the vocabulary) at most 2e-5 of the logits' root mean square; bfloat16: at most 4e-2 of it for at least
nine rows in ten (a router choice that rounding flips is no fault)."""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Optional

import torch

from satapel_cases import assert_rows, oracle_view, row_errors, tokens  # noqa: F401  (the rules are the same)


def latent(heads, dim, rot_dim, vdim, q_rank, rank, scale, window=None, base=10000.0, mlp="dense"):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, scale, rot, softcap=None, window=None, base=10000.0, bands=None, mlp="dense"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if bands:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def moe(experts, top, ff, groups=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    return out


def model(width, vocab, layers, ff=48, eps=1e-6, scale=3.0, logit_scale=1.0, logit_softcap=0.0):
    out = []
    for layer in layers:
        layer = json.loads(json.dumps(layer))
        if layer["mlp"] == "dense":
            layer["mlp"] = {"kind": "dense", "ff": ff}
        out.append(layer)
    return {"architecture": "Nuvivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_scale": logit_scale, "logit_softcap": logit_softcap, "layers": out}


# latent first (three heads, a query latent narrower than the cached one, a window of 33); three query heads to a kv head,
# a third of a head rotated at banded frequencies (all three bands), a window of 70 (no multiple of a page), two of three
# groups of experts; a layer without a feed-forward; attention over every key with a soft-cap
CASE_A = model(72, 211, [latent(3, 16, 8, 24, 20, 40, 0.35, window=33),
                         attention(3, 1, 24, 16, 0.5, 8, softcap=4.0, window=70, base=100.0, bands=(8.0, 1.0, 4.0, 100),
                                   mlp=moe(6, 2, 40, groups=(3, 2))),
                         latent(2, 24, 4, 16, 56, 24, 0.3, window=64, mlp=None),
                         attention(4, 2, 8, 24, 0.9, 6, softcap=2.5, mlp=moe(5, 3, 16))],
               ff=56, logit_scale=0.7, logit_softcap=1.5)
# attention first; a window of one page and of one key; a kv head to every query head; a whole head rotated; no soft-caps;
# one expert of the one best group; one latent layer that sees every key
CASE_B = model(64, 150, [attention(2, 2, 8, 8, 0.7, 8, window=64, base=500.0, mlp=moe(4, 1, 24, groups=(2, 1))),
                         latent(4, 8, 16, 8, 32, 24, 0.4, base=500.0),
                         attention(4, 2, 16, 8, 0.4, 2, softcap=9.0, window=1, bands=(3.0, 0.5, 0.5, 40), mlp=None),
                         latent(1, 32, 16, 40, 8, 32, 0.25, window=1)],
               ff=40, eps=1e-5, scale=1.0, logit_scale=3.0, logit_softcap=8.0)
# every group kept; groups of one expert; values wider than keys; more heads than a block of the latent kernel takes
CASE_C = model(80, 90, [latent(9, 8, 4, 16, 24, 36, 0.4, window=100, mlp=moe(6, 4, 24, groups=(2, 2))),
                        attention(8, 1, 40, 48, 0.3, 12, softcap=3.0, window=10, base=50.0, bands=(2.0, 0.25, 2.0, 64)),
                        attention(6, 2, 8, 8, 0.8, 4, softcap=6.0, mlp=moe(4, 2, 16, groups=(4, 3))),
                        latent(2, 16, 2, 8, 40, 20, 0.5, window=17, base=50.0)], ff=24, scale=9.0)
# sizes that are multiples of nothing (a width of 100 is no multiple of 8: the tensor-core products step aside)
CASE_D = model(100, 77, [latent(5, 12, 6, 20, 26, 30, 0.3, window=45, mlp=moe(7, 3, 36)),
                         attention(5, 5, 10, 20, 0.6, 6, softcap=5.0, window=33, base=77.0, bands=(4.0, 1.5, 3.0, 50)),
                         latent(3, 10, 2, 6, 7, 18, 0.6, mlp=moe(9, 2, 12, groups=(3, 1)))],
               ff=36, eps=3e-5, scale=2.5, logit_scale=1.5, logit_softcap=4.0)
# wider layers: heads of 64 and 128 numbers (the tensor-core attention kernels), a window longer than four pages, a latent
# of 200 numbers with 16 heads (two head groups), experts and feed-forwards of several tiles
CASE_E = model(256, 500, [attention(8, 2, 64, 128, 0.15, 32, softcap=5.0, window=300, base=1000.0, bands=(4.0, 1.0, 4.0, 400),
                                    mlp=moe(8, 2, 264, groups=(4, 2))),
                          latent(16, 16, 16, 24, 136, 200, 0.25, window=290),
                          attention(4, 4, 128, 64, 0.1, 128, softcap=20.0, mlp=None),
                          latent(4, 32, 16, 40, 72, 200, 0.2, window=64, mlp=moe(12, 3, 72, groups=(3, 2)))],
               ff=520, logit_scale=0.4, logit_softcap=2.0)
CASES = {"A": (CASE_A, 81), "B": (CASE_B, 82), "C": (CASE_C, 83), "D": (CASE_D, 84), "E": (CASE_E, 85)}


def _scaled(name: str, t: torch.Tensor) -> torch.Tensor:
    t = t.float()
    if name.endswith(("norm1", "norm2", "final.norm", "dq.norm", "dkv.norm")):
        return 1.0 + t
    if name == "embed":
        return t * 25.0
    if name == "head":
        return t * 10.0
    if name.endswith(("mix.q", "mix.k", "mix.dq", "mix.dkv")):
        return t * 6.0
    if name.endswith((".q.b", ".k.b", ".v.b")):
        return t * 6.0
    if name.endswith("sink"):
        return 1.0 + t
    if name.endswith("router"):
        return t * 0.5
    if name.endswith(("uq", ".up", ".down", "mix.uk", "mix.uv", "mix.v", "mix.o")):
        return t * 3.0
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
