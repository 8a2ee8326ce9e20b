"""Nuvivik in plain, slow PyTorch (float64 by default, whole sequences, loops): the oracle of the tests.

One function per mechanism, written from the design's equations; nothing here is shared with the
library.  A model is (cfg, w): cfg the dict that config.json holds, w a dict of tensors by
checkpoint name.

  rms                 x / sqrt(mean(x^2) + eps)
  frequencies         base^(-2i/dims); with a scaling: unchanged for short wavelengths, divided by the
                      factor for long ones, a straight line between the two in original / wavelength
  rotate_halves       rotary positions on pairs (i, i + dims/2) of the first `dims` numbers
  capped              c tanh(s / c); no cap: s
  visible             the mask: causal, the last `size` keys
  latent_mixer        queries from a normed latent, keys and values expanded from one normed latent row per
                      position, one rotated key part shared by the heads, one more term in the denominator
  attention_mixer     grouped queries with biases; rotation, then q and k over their root mean square; a
                      soft-capped score
  dense_ff            down(gelu(up h)), the tanh form
  choose              the experts a token uses: the largest scores among the experts of the best groups
  routed_ff           the chosen experts' down(relu(up h)^2), weighted with their scores as they are
  forward             per layer: x += norm1(mixer(x)); x += norm2(ff(x)), the branches reading x itself
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot) -> List[float]:
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_halves(vec, pos: int, rot):
    """vec [..., n]: the first rot.dims numbers rotated, number i with number i + dims/2."""
    dims = rot["dims"]
    half = dims // 2
    a = pos * torch.tensor(frequencies(rot), dtype=vec.dtype)
    c, s = torch.cos(a), torch.sin(a)
    out = vec.clone()
    u, v = vec[..., :half], vec[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def visible(i: int, j: int, mask: Optional[dict]) -> bool:
    return j <= i and (not mask or i - j < mask["size"])


def softmax_with_sink(s, sink=None):
    """Weights over s; `sink` (one number) joins the denominator as exp(sink)."""
    top = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - top)
    return e / (e.sum() + (0.0 if sink is None else torch.exp(sink - top)))


def capped(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def latent_mixer(m, eps, w, p, h):
    T, H, d, r, vd, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :R], eps) * w[p + "dkv.norm"]
    kr = torch.stack([rotate_halves(down[t, R:], t, m["rot"]) for t in range(T)])
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, vd)
    out = torch.zeros(T, H, vd, dtype=h.dtype)
    for i in range(T):
        js = torch.tensor([j for j in range(T) if visible(i, j, m.get("mask"))])
        for hd in range(H):
            s = (k[js, hd] @ q[i, hd, :d] + kr[js] @ rotate_halves(q[i, hd, d:], i, m["rot"])) * m["scale"]
            out[i, hd] = softmax_with_sink(s, w[p + "sink"][hd]) @ v[js, hd]
    return out.reshape(T, H * vd) @ w[p + "o"].T


def attention_mixer(m, eps, w, p, h):
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, vd)
    q = torch.stack([rms(rotate_halves(q[t], t, m["rot"]), eps) for t in range(T)])
    k = torch.stack([rms(rotate_halves(k[t], t, m["rot"]), eps) for t in range(T)])
    out = torch.zeros(T, H, vd, dtype=h.dtype)
    for i in range(T):
        js = torch.tensor([j for j in range(T) if visible(i, j, m.get("mask"))])
        for hd in range(H):
            g = hd // (H // G)
            s = (k[js, g] @ q[i, hd]) * m["scale"]
            out[i, hd] = softmax_with_sink(capped(s, m.get("softcap"))) @ v[js, g]
    return out.reshape(T, H * vd) @ w[p + "o"].T


def dense_ff(w, p, h):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def expert_ff(w, p, h):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def choose(router, s) -> List[int]:
    """The experts for one token's scores s."""
    n = len(s)
    open_ = list(range(n))
    if router.get("groups"):
        count, keep = router["groups"]["count"], router["groups"]["keep"]
        size = n // count
        of_group = [sum(sorted((float(v) for v in s[g * size:(g + 1) * size]), reverse=True)[:2]) for g in range(count)]
        best = sorted(range(count), key=lambda g: (-of_group[g], g))[:keep]
        open_ = [e for e in open_ if e // size in best]
    return sorted(open_, key=lambda e: (-float(s[e]), e))[:router["top"]]


def routed_ff(mlp, w, p, h):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        s = torch.sigmoid(w[p + "router"] @ h[t])
        for e in choose(mlp["router"], s):
            out[t] += s[e] * expert_ff(w, f"{p}e{e}.", h[t])
    return out


def feed_forward(mlp, w, p, h):
    return dense_ff(w, p, h) if mlp["kind"] == "dense" else routed_ff(mlp, w, p, h)


def forward(cfg, w, tokens: List[int], taps: Optional[list] = None, edit=None):
    """Logits [T, vocab] of one sequence.  `taps`, a list, receives the residual stream after every layer.
    `edit(layer index, mixer constants)` may return a changed copy of a mixer's constants (tests use it to move a
    window's edge)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = layer["mixer"] if edit is None else edit(i, dict(layer["mixer"]))
        mixer = latent_mixer if layer["type"] == "latent_attention" else attention_mixer
        x = x + rms(mixer(m, eps, w, p + "mix.", x), eps) * w[p + "norm1"]
        if layer.get("mlp") is not None:
            x = x + rms(feed_forward(layer["mlp"], w, p + "mlp.", x), eps) * w[p + "norm2"]
        if taps is not None:
            taps.append(x.clone())
    return capped((rms(x, eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"], cfg["logit_softcap"])
