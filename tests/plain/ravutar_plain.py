"""Ravutar in plain, slow PyTorch (float64 by default, whole sequences, loops): the oracle of the tests.

One function per mechanism, written from the design's equations; nothing here is shared with the
library.  A model is (cfg, w): cfg the dict that config.json holds, w a dict of tensors by
checkpoint name.

  rms               x / sqrt(mean(x^2) + eps)
  gelu              0.5 x (1 + erf(x / sqrt 2))
  short_conv        y_t[c] = sum_j w[c, j] u_(t - taps + 1 + j)[c], zeros before the start
  query_factor      1 + coef ln(floor((p + 1) / every) + 1)
  softmax_branch    attention with grouped queries, biases, short convolutions on q, k, v, a query factor by
                    position, a one in the softmax's denominator
  channel_decay     logistic(W_a2 W_a1 h + b)^(1 / tau), one number per key channel
  gated_linear      S <- diag(alpha) S + k v^T, o = S^T q; head norm, silu gate
  parallel_mixer    left_scale * softmax_branch + right_scale * gated_linear
  mamba2_mixer      S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x; gate, then a norm in equal parts
  dense_ff          W_down gelu(W_up h + b) + b
  sublayer          the hyper-connections: `streams` copies of x, mixed, and the branch's output added to each
  forward           the run order with its loop
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu(x):
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


def short_conv(u, wc):
    """u [T, C], wc [C, taps], the last tap the current token's."""
    T, C = u.shape
    taps = wc.shape[1]
    out = torch.zeros(T, C, dtype=u.dtype)
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += wc[:, j] * u[src]
    return out


def query_factor(q_temp: Optional[dict], pos: int) -> float:
    if not q_temp:
        return 1.0
    return 1.0 + q_temp["coef"] * math.log((pos + 1) // q_temp["every"] + 1)


def softmax_branch(m, w, p, h):
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    def channels(name):             # a layer whose constants name no taps has no convolution
        u = h @ w[p + name].T + w[p + name + ".b"]
        return short_conv(u, w[p + name + ".conv"]) if m.get("conv") else u
    q, k, v = channels("q").view(T, H, d), channels("k").view(T, G, d), channels("v").view(T, G, vd)
    out = torch.zeros(T, H, vd, dtype=h.dtype)
    for i in range(T):
        lo = max(0, i + 1 - m["only_last"]) if m.get("only_last") else 0      # a test may take far keys away
        for hd in range(H):
            g = hd // (H // G)
            s = (k[lo:i + 1, g] @ (q[i, hd] * query_factor(m.get("q_temp"), i))) * m["scale"]
            top = max(float(s.max()), 0.0)
            e = torch.exp(s - top)
            one = math.exp(-top) if not m.get("no_sink") else 0.0
            out[i, hd] = (e / (one + e.sum())) @ v[lo:i + 1, g]
    return out.reshape(T, H * vd) @ w[p + "o"].T + w[p + "o.b"]


def channel_decay(m, w, p, h):
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return torch.exp(torch.nn.functional.logsigmoid(z) / m["tau"]).view(h.shape[0], m["heads"], m["dim"])


def gated_linear(m, eps, w, p, h):
    T, H, d, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, vd)
    alpha = channel_decay(m, w, p, h)
    out = torch.zeros(T, H, vd, dtype=h.dtype)
    for hd in range(H):
        S = torch.zeros(d, vd, dtype=h.dtype)
        for t in range(T):
            S = alpha[t, hd][:, None] * S + torch.outer(k[t, hd], v[t, hd])
            out[t, hd] = rms(S.T @ q[t, hd], eps) * w[p + "norm"]
    return (out.reshape(T, H * vd) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(m, eps, w, p, h):
    return m["left_scale"] * softmax_branch(m["left"], w, p + "left.", h) \
        + m["right_scale"] * gated_linear(m["right"], eps, w, p + "right.", h)


def mamba2_mixer(m, eps, w, p, h):
    T, H, vd, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    row = h @ w[p + "in"].T
    z, u, dt = row[:, :inner], row[:, inner:2 * inner + 2 * G * N], row[:, 2 * inner + 2 * G * N:]
    u = silu(short_conv(u, w[p + "conv"]) + w[p + "conv.b"])
    x, B, C = u[:, :inner].view(T, H, vd), u[:, inner:inner + G * N].view(T, G, N), u[:, inner + G * N:].view(T, G, N)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=1e9)
    y = torch.zeros(T, H, vd, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        a = torch.exp(w[p + "A_log"][hd])
        S = torch.zeros(N, vd, dtype=h.dtype)
        for t in range(T):
            S = torch.exp(-a * dt[t, hd]) * S + dt[t, hd] * torch.outer(B[t, g], x[t, hd])
            y[t, hd] = S.T @ C[t, g] + w[p + "D"][hd] * x[t, hd]
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def dense_ff(w, p, h):
    return gelu(h @ w[p + "up"].T + w[p + "up.b"]) @ w[p + "down"].T + w[p + "down.b"]


def sublayer(X, w, p, norm_w, eps, branch):
    """X [streams, T, width] -> the new streams.  mix is [from, to]."""
    s = X.shape[0]
    u = sum(w[p + "in"][a] * X[a] for a in range(s))
    y = branch(rms(u, eps) * norm_w)
    return torch.stack([sum(w[p + "mix"][a, t] * X[a] for a in range(s)) + w[p + "out"][t] * y for t in range(s)])


def run_order(cfg) -> List[int]:
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, w, tokens: List[int], taps: Optional[list] = None, edit=None, order: Optional[List[int]] = None):
    """Logits [T, vocab] of one sequence.  `taps`, a list, receives the sum of the streams after every layer run.
    `edit(layer index, mixer constants)` may return a changed copy of a mixer's constants; `order` replaces the run
    order (tests use both to see that a mechanism matters)."""
    eps = cfg["norm"]["eps"]
    X = torch.stack([w["embed"][torch.tensor(tokens)]] * cfg["streams"])
    for i in run_order(cfg) if order is None else order:
        layer, p = cfg["layers"][i], f"l{i}."
        m = layer["mixer"] if edit is None else edit(i, dict(layer["mixer"]))
        mix = parallel_mixer if layer["type"] == "parallel" else mamba2_mixer
        X = sublayer(X, w, p + "hc1.", w[p + "norm1"], eps, lambda h: mix(m, eps, w, p + "mix.", h))
        if layer.get("mlp") is not None:
            X = sublayer(X, w, p + "hc2.", w[p + "norm2"], eps, lambda h: dense_ff(w, p + "mlp.", h))
        if taps is not None:
            taps.append(X.sum(0))
    return (rms(X.sum(0), eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]
