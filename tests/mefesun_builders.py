"""Small random Mefesun models for tests: configurations, weights on the bf16 grid, and models whose weights make one mechanism
stand out."""
import numpy as np

from ratchet_b200 import capi

from .dadezen_builders import YARN, write_model  # noqa: F401  (one place for both families)


def attention(heads, kv_heads, dim, vdim, chunk, scale, dims=None, base=10000.0, scaling=None, ff=None, weights_of=None):
    rot = {"base": base, "dims": dim if dims is None else dims}
    if scaling:
        rot["scaling"] = scaling
    e = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "scale": scale, "rot": rot},
         "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(width, vocab, layers, softcap=20.0, eps=1e-5):
    c = {"architecture": "Mefesun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}
    if softcap:
        c["logit_softcap"] = softcap
    return c


def on_grid(W):
    return {k: capi.from_bf16(capi.to_bf16(np.asarray(v, np.float32))) for k, v in W.items()}


def weights(cfg, seed, head_gain=1.6):
    """Random tensors whose values bf16 holds exactly.  The head norms are scaled up so that single keys stand out of the softmax, and
    the sinks are of the size of the scores."""
    g = np.random.Generator(np.random.PCG64(seed))
    W, d = {}, cfg["width"]

    def mat(name, rows, cols):
        W[name] = g.standard_normal((rows, cols)) / np.sqrt(cols)

    def vec(name, n, mean=0.0, spread=0.3):
        W[name] = mean + spread * g.standard_normal(n)

    W["embed"] = g.standard_normal((cfg["vocab"], d)) + 0.3
    vec("final.norm", d, 1.0)
    vec("final.norm.b", d)
    for i, e in enumerate(cfg["layers"]):
        if e.get("weights_of") is not None:
            continue
        m, p, x = e["mixer"], f"l{i}.", f"l{i}.mix."
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * E)):
            mat(x + n, rows, d)
            vec(x + n + ".b", rows)
        vec(x + "q.norm", D, head_gain)
        vec(x + "k.norm", D, head_gain)
        vec(x + "sink", H, 2.0, 1.5)
        mat(x + "o", d, H * E)
        vec(x + "o.b", d)
        for k in "12" if e["mlp"] else "1":
            vec(f"{p}norm{k}", d, 1.0)
            vec(f"{p}norm{k}.b", d)
            vec(f"{p}ls{k}", d, 0.8)
        if e["mlp"]:
            mat(p + "mlp.up", e["mlp"]["ff"], d)
            mat(p + "mlp.down", d, e["mlp"]["ff"])
    return on_grid(W)


# Sizes that are awkward for the kernels on purpose: heads and features that are no multiples of 8, single heads and as many key heads as
# query heads, more query heads per key head than a tensor-core tile holds, chunks of one position, layers without a feed-forward,
# layers that share weights, chunks of different sizes in one model.
CONFIGS = {
    "mixed": config(80, 91, [attention(6, 2, 24, 40, 37, 0.2, dims=16, scaling=YARN, ff=112), attention(4, 4, 16, 16, 5, 0.25, base=500.0),
                             attention(6, 2, 24, 40, 37, 0.2, dims=16, scaling=YARN, ff=112, weights_of=0),
                             attention(5, 1, 32, 24, 64, 0.15, scaling=YARN, ff=48),
                             attention(6, 2, 24, 40, 37, 0.2, dims=16, scaling=YARN, ff=112, weights_of=2)]),
    "odd": config(45, 53, [attention(3, 1, 5, 7, 11, 0.4, dims=4, scaling=YARN, ff=31), attention(2, 2, 9, 3, 1, 0.3, dims=2), attention(1, 1, 9, 13, 150, 0.3, dims=8, ff=17)],
                  softcap=None, eps=1e-3),
    "many": config(64, 70, [attention(20, 1, 32, 32, 70, 0.12, scaling=YARN, ff=96), attention(36, 2, 16, 24, 129, 0.2, dims=8, ff=64)], softcap=6.0),
    "wide": config(160, 130, [attention(4, 2, 128, 128, 130, 0.07, base=50000.0, scaling=YARN, ff=200), attention(2, 1, 200, 136, 300, 0.05, dims=64, ff=136),
                              attention(2, 2, 40, 264, 48, 0.1, dims=24)]),
}


def loud_case(chunk, heads=4, kv_heads=2, dim=16, vdim=16, dims=8):
    """A one-layer model in which token 1's key scores far above every other key for all queries (through features that are not rotated)
    and carries a value of its own; the other tokens' keys score alike.  Whether position i sees a loud position decides its logits."""
    g = np.random.Generator(np.random.PCG64(chunk + 1000 * dim))
    d, vocab = 48, 40
    cfg = config(d, vocab, [attention(heads, kv_heads, dim, vdim, chunk, 1.5, dims=dims)], softcap=None)
    W = weights(cfg, 3)
    W["embed"] = 0.3 * g.standard_normal((vocab, d))
    W["embed"][:, 0] = -4.0
    W["embed"][:, 1] = 0.0
    W["embed"][1, :2] = (4.0, 6.0)
    W["final.norm"][:2] = W["final.norm.b"][:2] = 0.0      # the logits ignore the two features that mark the token
    x, u = "l0.mix.", np.zeros(dim)
    u[dims:] = 1.0                                    # the features that are not rotated
    W[x + "q"] = 0.02 * W[x + "q"]
    W[x + "q.b"] = np.tile(2.0 * u, heads)
    W[x + "k"] = 0.02 * W[x + "k"]
    W[x + "k"][:, 0] = np.tile(u, kv_heads)
    W[x + "k.b"] = np.zeros(kv_heads * dim)
    W[x + "v"] = 0.1 * W[x + "v"]
    W[x + "v"][:, 1] = np.resize([1.0, -1.0, 0.5], kv_heads * vdim)
    W[x + "q.norm"] = W[x + "k.norm"] = np.ones(dim)
    W[x + "sink"] = np.full(heads, -4.0)
    return cfg, on_grid(W)
