"""Small random Dadezen models for tests: configurations, weights on the bf16 grid, and folders on disk."""
import json
import os

import numpy as np

from ratchet_b200 import capi


def lightning(heads, dim, vdim, decay, ff=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, scale, base=10000.0, dims=None, scaling=None, ff=None):
    rot = {"base": base, "dims": rot_dim if dims is None else dims}
    if scaling:
        rot["scaling"] = scaling
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "mask": {"size": window}, "scale": scale, "rot": rot},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, loop=None, mult=0.7, eps=1e-5):
    c = {"architecture": "Dadezen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed, attention_gain=1.5):
    """Random tensors whose values bf16 holds exactly.  Queries and keys of the attention layers are scaled up so that single
    keys stand out of the softmax."""
    g = np.random.Generator(np.random.PCG64(seed))
    W, d = {}, cfg["width"]

    def mat(name, rows, cols, gain=1.0):
        W[name] = gain * g.standard_normal((rows, cols)) / np.sqrt(cols)

    def scale(name, n):
        W[name] = 1.0 + 0.2 * g.standard_normal(n)

    W["embed"] = g.standard_normal((cfg["vocab"], d)) + 0.3
    mat("head", cfg["vocab"], d)
    scale("final.norm", d)
    if cfg.get("loop"):
        mat("loop.in", d, 2 * d)
        W["loop.step"] = 0.5 * g.standard_normal((cfg["loop"]["times"], d))
    for i, e in enumerate(cfg["layers"]):
        m, x = e["mixer"], f"l{i}.mix."
        H, D, E = m["heads"], m["dim"], m["vdim"]
        scale(f"l{i}.norm1", d)
        if e["type"] == "lightning":
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * E), ("g", H * E)):
                mat(x + n, rows, d, 1.5)
            scale(x + "norm", H * E)
        else:
            Q, C, R = m["q_rank"], m["kv_rank"], m["rot_dim"]
            mat(x + "dq", Q, d)
            scale(x + "dq.norm", Q)
            mat(x + "uq", H * (D + R), Q, attention_gain)
            mat(x + "dkv", C + R, d)
            scale(x + "dkv.norm", C)
            mat(x + "uk", H * D, C, attention_gain)
            mat(x + "uv", H * E, C)
        mat(x + "o", d, H * E)
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            scale(f"l{i}.norm2", d)
            mat(f"l{i}.mlp.gate", ff, d)
            mat(f"l{i}.mlp.up", ff, d)
            mat(f"l{i}.mlp.down", d, ff)
    return {k: capi.from_bf16(capi.to_bf16(v.astype(np.float32))) for k, v in W.items()}


def write_safetensors(path, tensors):
    """tensors: name -> (dtype name, array of the stored bits)."""
    header, at, blobs = {}, 0, []
    for name, (dt, a) in tensors.items():
        b = np.ascontiguousarray(a).tobytes()
        header[name] = {"dtype": dt, "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    h = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h + b"".join(blobs))


def write_model(folder, cfg, W):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: ("BF16", capi.to_bf16(v)) for k, v in W.items()})
    return str(folder)


YARN = {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.0}

# Sizes that are awkward for the kernels on purpose: heads, features and ranks that are no multiples of 8 or 16, single heads,
# windows of one token, loops over one layer, layers without a feed-forward.
CONFIGS = {
    "mixed": config(80, 91, [lightning(3, 24, 40, (0.3, 0.9, 0.998), ff=112), latent(5, 16, 8, 24, 48, 64, 37, 0.2, scaling=YARN, ff=72),
                             latent(2, 32, 16, 16, 40, 56, 5, 0.15, base=500.0, ff=48), lightning(2, 16, 16, (0.75, 0.97))], loop=(1, 3, 2)),
    "odd": config(45, 53, [latent(3, 5, 6, 7, 19, 21, 11, 0.3, dims=4, scaling=YARN), lightning(1, 9, 13, (0.95,), ff=31),
                           latent(1, 8, 2, 9, 10, 12, 1, 0.5, ff=17)], loop=(0, 1, 3), mult=1.0),
    "plain": config(64, 70, [lightning(4, 32, 32, (0.5, 0.8, 0.99, 1.0), ff=96), latent(3, 40, 24, 48, 64, 96, 70, 0.11, scaling=YARN, ff=96)], mult=0.4),
    "wide": config(160, 130, [latent(3, 128, 64, 128, 96, 144, 130, 0.07, base=50000.0, dims=64, scaling=YARN, ff=200),
                              lightning(2, 128, 128, (0.9, 0.99), ff=256)], loop=(1, 2, 2)),
}
