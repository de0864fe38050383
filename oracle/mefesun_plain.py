"""Plain restatement of the Mefesun language model in numpy float64: one function per mechanism, nothing shared with the
product path.  Test infrastructure only.

x is the residual stream [T, width]; linear weights are [out, in]; positions are absolute and start at 0; attention takes the
whole history.  Functions of mechanisms that the two plain models share come from dadezen_plain.
"""
from __future__ import annotations

import math

import numpy as np

from .dadezen_plain import linear, rms_norm, rotate


def layer_norm_bias(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w + b


def squared_relu(z):
    return np.where(z > 0, z, 0.0) ** 2


def softcap(z, cap):
    return z if cap is None else cap * np.tanh(z / cap)


def same_chunk(i, j, size):
    """Does position i see position j <= i when attention stays inside chunks of `size` positions?  (None: always.)"""
    return j <= i and (size is None or i // size == j // size)


def sink_attention(q, k, v, scale, sink, size):
    """q [T, H, D], k [T, G, D], v [T, G, E]; query head h reads key head h // (H / G).  exp(sink[h]) joins the denominator."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    o = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        seen = [j for j in range(i + 1) if same_chunk(i, j, size)]
        for h in range(H):
            s = k[seen, h // per] @ q[i, h] * scale
            top = max(s.max(), sink[h])
            p = np.exp(s - top)
            o[i, h] = p @ v[seen, h // per] / (p.sum() + math.exp(sink[h] - top))
    return o


def attention_mixer(W, pre, h, cfg, eps):
    T, H, G, D, E = len(h), cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    proj = lambda n: linear(W[pre + n], h) + W[pre + n + ".b"]
    q = rms_norm(proj("q").reshape(T, H, D), W[pre + "q.norm"], eps)
    k = rms_norm(proj("k").reshape(T, G, D), W[pre + "k.norm"], eps)
    v = proj("v").reshape(T, G, E)
    pos = np.arange(T)
    o = sink_attention(rotate(q, pos, cfg["rot"]), rotate(k, pos, cfg["rot"]), v, cfg["scale"], W[pre + "sink"],
                       cfg["mask"]["size"] if cfg.get("mask") else None)
    return linear(W[pre + "o"], o.reshape(T, H * E)) + W[pre + "o.b"]


def feed_forward(W, pre, h):
    return linear(W[pre + "down"], squared_relu(linear(W[pre + "up"], h)))


def owner(config, i):
    """The layer whose tensors layer i uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def layer(W, p, entry, x, eps):
    out = attention_mixer(W, p + "mix.", x, entry["mixer"], eps)
    x = x + W[p + "ls1"] * layer_norm_bias(out, W[p + "norm1"], W[p + "norm1.b"], eps)
    if entry.get("mlp"):
        out = feed_forward(W, p + "mlp.", x)
        x = x + W[p + "ls2"] * layer_norm_bias(out, W[p + "norm2"], W[p + "norm2.b"], eps)
    return x


def forward(config, W, tokens, streams=None):
    """Logits [T, vocab] of a whole prompt.  `streams`, if given, receives the residual stream after every layer."""
    W = {k: np.asarray(v, np.float64) for k, v in W.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    for i, entry in enumerate(config["layers"]):
        x = layer(W, f"l{owner(config, i)}.", entry, x, eps)
        if streams is not None:
            streams.append(x.copy())
    z = linear(W["embed"], layer_norm_bias(x, W["final.norm"], W["final.norm.b"], eps))
    return softcap(z, config.get("logit_softcap"))
