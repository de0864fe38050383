"""Plain restatement of the Dadezen language model in numpy float64: one function per mechanism, token loops where
the mechanism is sequential, no caching tricks, nothing shared with the product path.  Test infrastructure only.

Notation: x is the residual stream [T, width]; h is a normalised copy of it; every linear map stores its weight as
[out, in].  Positions are absolute and start at 0; functions that attend or recur take the whole history.
"""
from __future__ import annotations

import math

import numpy as np


def linear(w, h):
    return h @ np.asarray(w, np.float64).T


def layer_norm(x, w, eps):
    """Weight, no bias; the variance is the mean squared deviation from the row mean."""
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_mlp(h, gate, up, down):
    return linear(down, gelu_tanh(linear(gate, h)) * linear(up, h))


def rotary_frequencies(rot):
    """Angular frequency of every pair and the factor on cos and sin (1 without YaRN scaling)."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return np.array(f), 1.0

    def at(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(at(sc["fast"])), 0)
    hi = min(math.ceil(at(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1.0 - r))
    return np.array(out), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(v, positions, rot):
    """Interleaved pairs (2i, 2i+1) of the first rot['dims'] entries of the last axis; v is [T, ..., D]."""
    f, m = rotary_frequencies(rot)
    v = np.array(v, np.float64)
    for t, p in enumerate(positions):
        for i in range(rot["dims"] // 2):
            c, s = m * math.cos(p * f[i]), m * math.sin(p * f[i])
            a, b = v[t, ..., 2 * i].copy(), v[t, ..., 2 * i + 1].copy()
            v[t, ..., 2 * i] = a * c - b * s
            v[t, ..., 2 * i + 1] = b * c + a * s
    return v


def linear_attention(q, k, v, decay, state=None):
    """q, k [T, H, D], v [T, H, E]: S <- decay_h S + k v^T, o = S^T q.  Returns o [T, H, E] and the last S."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else np.array(state, np.float64)
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def lightning_mixer(W, pre, h, cfg, eps):
    T, H, D, E = len(h), cfg["heads"], cfg["dim"], cfg["vdim"]
    q = silu(linear(W[pre + "q"], h)).reshape(T, H, D)
    k = silu(linear(W[pre + "k"], h)).reshape(T, H, D)
    v = silu(linear(W[pre + "v"], h)).reshape(T, H, E)
    o, _ = linear_attention(q, k, v, cfg["decay"])
    y = rms_norm(o.reshape(T, H * E), W[pre + "norm"], eps) * sigmoid(linear(W[pre + "g"], h))
    return linear(W[pre + "o"], y)


def windowed_softmax_attention(q, k, v, scale, window):
    """q, k [T, H, D], v [T, H, E]; position i sees i - window < j <= i."""
    T, H, _ = q.shape
    o = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        j0 = max(0, i - window + 1)
        for h in range(H):
            s = k[j0:i + 1, h] @ q[i, h] * scale
            p = np.exp(s - s.max())
            o[i, h] = (p / p.sum()) @ v[j0:i + 1, h]
    return o


def latent_mixer(W, pre, h, cfg, eps):
    T, H, D, R, E, C = len(h), cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    pos = np.arange(T)
    q = linear(W[pre + "uq"], rms_norm(linear(W[pre + "dq"], h), W[pre + "dq.norm"], eps)).reshape(T, H, D + R)
    q = np.concatenate([q[..., :D], rotate(q[..., D:], pos, cfg["rot"])], -1)
    low = linear(W[pre + "dkv"], h)
    c = rms_norm(low[:, :C], W[pre + "dkv.norm"], eps)
    kr = rotate(low[:, C:], pos, cfg["rot"])
    k = linear(W[pre + "uk"], c).reshape(T, H, D)
    k = np.concatenate([k, np.repeat(kr[:, None, :], H, 1)], -1)
    v = linear(W[pre + "uv"], c).reshape(T, H, E)
    o = windowed_softmax_attention(q, k, v, cfg["scale"], cfg["mask"]["size"])
    return linear(W[pre + "o"], o.reshape(T, H * E))


MIXERS = {"lightning": lightning_mixer, "latent_attention": latent_mixer}


def layer_order(config):
    """(layer, pass) of every layer run; pass is None outside the loop."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    run = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        run += [(i, t) for i in range(loop["start"], loop["stop"])]
    return run + [(i, None) for i in range(loop["stop"], n)]


def layer(W, i, entry, x, config):
    eps = config["norm"]["eps"]
    pre = f"l{i}."
    out = MIXERS[entry["type"]](W, pre + "mix.", layer_norm(x, W[pre + "norm1"], eps), entry["mixer"], eps)
    if entry.get("mlp"):
        h = layer_norm(x, W[pre + "norm2"], eps)
        out = out + gated_mlp(h, W[pre + "mlp.gate"], W[pre + "mlp.up"], W[pre + "mlp.down"])
    return x + config["residual_mult"] * out


def forward(config, W, tokens, streams=None):
    """Logits [T, vocab] of a whole prompt.  `streams`, if given, receives the residual stream after every layer run."""
    W = {k: np.asarray(v, np.float64) for k, v in W.items()}
    x0 = W["embed"][np.asarray(tokens)]
    x = x0.copy()
    loop = config.get("loop")
    for i, t in layer_order(config):
        if t is not None and i == loop["start"]:
            x = linear(W["loop.in"], np.concatenate([x, x0], -1)) + W["loop.step"][t]
        x = layer(W, i, config["layers"][i], x, config)
        if streams is not None:
            streams.append(x.copy())
    return linear(W["head"], layer_norm(x, W["final.norm"], config["norm"]["eps"]))
