"""`python bench.py --serve`: prefill and decode throughput of the Mefesun decoder (grouped heads of 128, four query heads per key head,
chunks as long as the window) and the Dadezen decoder (half of the layers linear attention, half windowed latent attention) at
layer sizes of real models with random bf16 weights, beside Phi-3's layers at the same width, feed-forward and depth (f16 prefill
through the lazy graph, Q8_0 decode through the fused step).

One JSON line: per size and model the tokens per second, the share of the measured roofline (weights and states once per decoded token
over the copy bandwidth; matrix-product flops of a prompt over the sustained tensor throughput) and, per op of the lazy graph, its
time and the share of its own roofline."""
from __future__ import annotations

import json

import numpy as np

SIZES = {
    "w1024": dict(width=1024, ff=2816, layers=8, vocab=32000, heads=8, dim=128, vdim=128, l_heads=8, l_dim=64, l_rot=32, l_vdim=64, q_rank=384, kv_rank=256,
                  window=512, prompt=2048),
    "w2048": dict(width=2048, ff=5632, layers=8, vocab=32000, heads=16, dim=128, vdim=128, l_heads=16, l_dim=128, l_rot=64, l_vdim=128, q_rank=768,
                  kv_rank=512, window=1024, prompt=4096),
    "w4096": dict(width=4096, ff=11008, layers=8, vocab=32000, heads=32, dim=128, vdim=128, l_heads=32, l_dim=128, l_rot=64, l_vdim=128, q_rank=1536,
                  kv_rank=512, window=2048, prompt=4096),
}


def dadezen_config(c):
    n = c["layers"] // 2
    decay = [float(1.0 - 2.0 ** -(2 + 6 * i / c["heads"])) for i in range(c["heads"])]
    pair = [{"type": "lightning", "mixer": {"heads": c["heads"], "dim": c["dim"], "vdim": c["vdim"], "decay": decay}, "mlp": {"kind": "dense", "ff": c["ff"]}},
            {"type": "latent_attention",
             "mixer": {"heads": c["l_heads"], "dim": c["l_dim"], "rot_dim": c["l_rot"], "vdim": c["l_vdim"], "q_rank": c["q_rank"], "kv_rank": c["kv_rank"],
                       "mask": {"size": c["window"]}, "scale": (c["l_dim"] + c["l_rot"]) ** -0.5,
                       "rot": {"base": 10000.0, "dims": c["l_rot"], "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}},
             "mlp": {"kind": "dense", "ff": c["ff"]}}]
    return {"architecture": "Dadezen", "width": c["width"], "vocab": c["vocab"], "norm": {"eps": 1e-5}, "residual_mult": 0.5, "layers": pair * n}


def mefesun_config(c):
    d = c["width"]
    layer = {"type": "attention", "mixer": {"heads": d // 128, "kv_heads": max(d // 512, 1), "dim": 128, "vdim": 128, "mask": {"size": c["window"]}, "scale": 128 ** -0.5,
                                            "rot": {"base": 10000.0, "dims": 128,
                                                    "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}},
             "mlp": {"kind": "dense", "ff": c["ff"]}}
    return {"architecture": "Mefesun", "width": d, "vocab": c["vocab"], "norm": {"eps": 1e-5}, "logit_softcap": 50.0, "layers": [layer] * c["layers"]}


def mefesun_shapes(config):
    d = config["width"]
    S = {"embed": (config["vocab"], d), "final.norm": (d,), "final.norm.b": (d,)}
    for i, e in enumerate(config["layers"]):
        m, ff, p, x = e["mixer"], e["mlp"]["ff"], f"l{i}.", f"l{i}.mix."
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * E)):
            S[x + n], S[x + n + ".b"] = (rows, d), (rows,)
        S.update({x + "o": (d, H * E), x + "o.b": (d,), x + "q.norm": (D,), x + "k.norm": (D,), x + "sink": (H,), p + "mlp.up": (ff, d), p + "mlp.down": (d, ff)})
        for k in "12":
            S[f"{p}norm{k}"] = S[f"{p}norm{k}.b"] = S[f"{p}ls{k}"] = (d,)
    return S


def mefesun_work(c):
    """As dadezen_work."""
    m, d, ff, n, T = mefesun_config(c)["layers"][0]["mixer"], c["width"], c["ff"], c["layers"], c["prompt"]
    H, G, D, E, W = m["heads"], m["kv_heads"], m["dim"], m["vdim"], min(c["window"], c["prompt"])
    weights = n * (d * (H * D + G * (D + E)) + H * E * d + 2 * d * ff) + d * c["vocab"]
    seen = T // W * (W * (W + 1) // 2) + (T % W) * (T % W + 1) // 2
    return 2 * weights + n * W * G * (D + E) * 2, {"linear": 2 * T * (weights - d * c["vocab"]), "grouped_attention": n * 2 * seen * H * (D + E)}


def dadezen_shapes(config):
    d, S = config["width"], {}
    S["embed"] = S["head"] = (config["vocab"], d)
    S["final.norm"] = (d,)
    for i, e in enumerate(config["layers"]):
        m, x, ff = e["mixer"], f"l{i}.mix.", e["mlp"]["ff"]
        H, D, E = m["heads"], m["dim"], m["vdim"]
        S[f"l{i}.norm1"] = S[f"l{i}.norm2"] = (d,)
        S[f"l{i}.mlp.gate"] = S[f"l{i}.mlp.up"] = (ff, d)
        S[f"l{i}.mlp.down"] = (d, ff)
        S[x + "o"] = (d, H * E)
        if e["type"] == "lightning":
            S.update({x + "q": (H * D, d), x + "k": (H * D, d), x + "v": (H * E, d), x + "g": (H * E, d), x + "norm": (H * E,)})
        else:
            Q, C, R = m["q_rank"], m["kv_rank"], m["rot_dim"]
            S.update({x + "dq": (Q, d), x + "dq.norm": (Q,), x + "uq": (H * (D + R), Q), x + "dkv": (C + R, d), x + "dkv.norm": (C,), x + "uk": (H * D, C),
                      x + "uv": (H * E, C)})
    return S


class RandomFile:
    """A weights file of random values (the loader's file interface)."""

    def __init__(self, shapes):
        from ratchet_b200 import capi
        self.shapes = shapes
        g = np.random.Generator(np.random.PCG64(3))
        self._pool = capi.to_bf16(g.standard_normal(1 << 22, dtype=np.float32) * np.float32(0.02))
        self._capi = capi

    def shape(self, name):
        return self.shapes[name]

    def __contains__(self, name):
        return name in self.shapes

    def raw(self, name):
        n = int(np.prod(self.shapes[name]))
        return "BF16", np.resize(self._pool, n).reshape(self.shapes[name])

    def f32(self, name):
        if len(self.shapes[name]) == 1:
            return np.ones(self.shapes[name], np.float32)
        return self._capi.from_bf16(self.raw(name)[1])


def dadezen_work(c):
    """(bytes per decoded token with a full window, matrix-product flops per prompt token, per-op flops of one prompt)."""
    d, ff, n, T = c["width"], c["ff"], c["layers"] // 2, c["prompt"]
    H, D, E = c["heads"], c["dim"], c["vdim"]
    h, ld, r, le, Q, C, W = c["l_heads"], c["l_dim"], c["l_rot"], c["l_vdim"], c["q_rank"], c["kv_rank"], min(c["window"], c["prompt"])
    mlp = 3 * d * ff
    lin = d * H * (2 * D + 2 * E) + H * E * d
    lat = d * (Q + C + r) + Q * h * (ld + r) + C * h * (ld + le) + h * le * d
    weights = n * (2 * mlp + lin + lat) + d * c["vocab"]
    decode = 2 * weights + n * (2 * H * D * E * 4 + W * (C + r) * 2)
    seen = (W * (W + 1) // 2 + (T - W) * W)                      # visible (query, key) pairs of the prompt
    flops = {"linear": 2 * T * n * (2 * mlp + lin + lat), "lightning": n * T * H * (4 * D * E + 128 * (D + E)),
             "window_attention": n * 2 * seen * h * (ld + r + le)}
    return decode, flops


def event_ms(torch, stream, fn, iters):
    for _ in range(3):
        fn()
    stream.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record(stream)
    for _ in range(iters):
        fn()
    b.record(stream)
    stream.synchronize()
    return a.elapsed_time(b) / iters


def op_table(dev, fn):
    """Per-op device time of one forward (event pair per node): op -> (count, us, GB/s over operand bytes)."""
    dev.set_debug(profile=True)
    dev.profile_report()
    fn()
    rows = {}
    for line in dev.profile_report().splitlines()[1:]:
        f = line.split()
        rows[" ".join(f[:-4])] = (int(f[-4]), float(f[-3]), float(f[-1]))
    dev.set_debug()
    return rows


NEW_MODELS = {"mefesun": (mefesun_config, mefesun_shapes, mefesun_work), "dadezen": (dadezen_config, dadezen_shapes, dadezen_work)}


def new_model_leg(dev, torch, stream, name, c, peaks, steps):
    from ratchet_b200 import Tensor
    from ratchet_b200.models import REGISTRY
    config, shapes, work = NEW_MODELS[name]
    cfg = config(c)
    m = REGISTRY[cfg["architecture"]](cfg, RandomFile(shapes(cfg)), dev)
    decode_bytes, flops = work(c)
    T = c["prompt"]
    ids = Tensor.from_data(np.random.Generator(np.random.PCG64(1)).integers(0, c["vocab"], T).astype(np.int32), device=dev)
    want = Tensor.from_data(np.array([T - 1], np.int32), device=dev)
    st = m.new_state()
    forward = lambda: m.graph.schedule(ids, st, want).resolve()
    prefill = event_ms(torch, stream, forward, 5)
    ops = op_table(dev, forward)
    # timed steps attend over a whole window, or the last hundred positions of a chunk
    if name == "mefesun":
        steps = min(steps, 100)
    st.position = T if name == "dadezen" else T - 1 - steps - 8
    m.decode(st, 5)
    decode = event_ms(torch, stream, lambda: m.decode(st), steps)
    gbs, tflops, sustained = peaks
    total = sum(flops.values())
    res = {"prompt_tokens": T, "prefill_tokens_per_s": T / prefill * 1e3, "prefill_ms": prefill, "prefill_tflops": total / prefill / 1e9,
           "prefill_frac": total / prefill / 1e9 / sustained,
           "decode_tokens_per_s": 1e3 / decode, "decode_us": decode * 1e3, "decode_bytes": decode_bytes,
           "decode_frac": decode_bytes / decode / 1e6 / gbs, "kernels_per_token": st.stack.kernels_per_step, "prefill_ops": {}}
    for k, (n, us, g) in ops.items():
        res["prefill_ops"][k] = {"count": n, "us": us, "gbs": g, "frac_of_bandwidth": g / gbs}
    for op, f in flops.items():                         # matrix products by op, whatever the output type
        us = sum(u for k, (_, u, _) in ops.items() if k.split()[0] == op)
        res["prefill_" + op] = {"us": us, "tflops": f / us / 1e6, "frac_of_tensor": f / us / 1e6 / tflops}
    dev.sync()
    return res


def phi3_leg(dev, torch, stream, c, peaks, steps):
    """Phi-3 layers of the same width, feed-forward and depth: heads of 128, a cache as long as the window."""
    from ratchet_b200 import Tensor, callers, capi, nn
    from ratchet_b200.decoder import Decoder, DecoderConfig, DecoderLayer
    d, ff, n, V, hd = c["width"], c["ff"], c["layers"], c["vocab"], 128
    H, T = d // 128, c["prompt"]
    g = np.random.Generator(np.random.PCG64(2))
    pool = (g.standard_normal(1 << 22, dtype=np.float32) * np.float32(0.02)).astype(np.float16)
    mat = lambda r, k: np.resize(pool, r * k).reshape(r, k)
    t = lambda a: Tensor.from_data(a, device=dev)
    ones = np.ones(d, np.float32)
    rope = nn.RotaryEmbedding(hd, False, 10000.0, 1.0)
    scale = t(np.array([hd ** -0.5], np.float32))
    layers = [callers.Phi3DecoderLayer(nn.RMSNorm(t(ones), 1e-5), callers.Phi3SelfAttention(nn.Linear(t(mat(3 * d, d))), nn.Linear(t(mat(d, d))), rope, H, H, scale),
                                       nn.RMSNorm(t(ones), 1e-5), callers.Phi3MLP(nn.Linear(t(mat(2 * ff, d))), nn.Linear(t(mat(d, ff))))) for _ in range(n)]
    model = callers.Phi3(nn.Embedding(t(mat(V, d))), layers, nn.RMSNorm(t(ones), 1e-5), nn.Linear(t(mat(V, d))), [None] * n)
    ids = t(g.integers(0, V, (1, T)).astype(np.int32))
    mask = t(np.triu(np.full((T, T), -65504.0, np.float16), 1))
    forward = lambda: model.schedule(ids, mask).resolve()
    prefill = event_ms(torch, stream, forward, 3)
    ops = op_table(dev, forward)
    linear = 2 * T * n * (4 * d * d + 3 * d * ff)
    attn = n * H * 2 * T * T * hd * 2                    # full products: the graph computes masked scores too
    del model, layers, mask
    from ratchet_b200.capi import Q8_0H
    raw = lambda r, k: dev.from_quantized(np.resize(g.integers(0, 127, 1 << 20).astype(np.uint8), capi.dtype_nbytes(Q8_0H, r * k)), Q8_0H, (r, k))
    cache, prior = c["window"] + 64, c["window"]
    dl = [DecoderLayer(dev.from_numpy(ones), raw(3 * d, d), raw(d, d), dev.from_numpy(ones), raw(2 * ff, d), raw(d, ff), dev.zeros(capi.F16, (H, cache, hd)),
                       dev.zeros(capi.F16, (H, cache, hd))) for _ in range(n)]
    dec = Decoder(dev, DecoderConfig(n, d, H, H, hd, ff, V, cache, hd, 10000.0, 1e-5, Q8_0H), dl, raw(V, d), dev.from_numpy(ones), raw(V, d))

    def step():
        dec.position = prior
        dec.step_device(argmax=False)
    dev.h2d(dec.token.ptr, np.array([7], np.int32))
    decode = event_ms(torch, stream, step, steps)
    elems = n * (4 * d * d + 3 * d * ff) + V * d
    b = int(elems * 1.0625) + n * 2 * H * prior * hd * 2
    gbs, tflops, sustained = peaks
    res = {"prompt_tokens": T, "prefill_tokens_per_s": T / prefill * 1e3, "prefill_ms": prefill, "prefill_tflops": (linear + attn) / prefill / 1e9,
           "prefill_frac": (linear + attn) / prefill / 1e9 / sustained,
           "decode_tokens_per_s": 1e3 / decode, "decode_us": decode * 1e3, "decode_bytes": b, "decode_frac": b / decode / 1e6 / gbs,
           "kernels_per_token": dec.kernels_per_step, "prefill_ops": {}}
    us = sum(u for k, (_, u, _) in ops.items() if k.split()[0] == "matmul")
    res["prefill_matmul"] = {"us": us, "tflops": (linear + attn) / us / 1e6, "frac_of_tensor": (linear + attn) / us / 1e6 / tflops}
    for k, (cnt, us, gb) in ops.items():
        res["prefill_ops"][k] = {"count": cnt, "us": us, "gbs": gb, "frac_of_bandwidth": gb / gbs}
    dec.close()
    dev.sync()
    return res


def run_serve(args, measured, clock_sampler):
    import torch

    from ratchet_b200 import Device
    torch.cuda.set_device(0)
    stream = torch.cuda.Stream()
    torch.cuda.set_stream(stream)
    dev = Device(0, stream=stream.cuda_stream)
    dev.set_constant_weights(True)
    peaks = (measured.get("hbm_gbs", 6650.0), measured.get("bf16_tflops", 1590.0), measured.get("bf16_tflops_sustained", 1400.0))
    sampler = clock_sampler(0)
    sampler.start()
    sizes = args.serve_sizes.split(",") if args.serve_sizes else list(SIZES)
    models = args.serve_models.split(",") if args.serve_models else list(NEW_MODELS)
    out = {}
    for name in sizes:
        c = SIZES[name]
        out[name] = {"config": c}
        for model in models:
            out[name][model] = new_model_leg(dev, torch, stream, model, c, peaks, args.steps)
            dev.check(dev._lib.rcu_pool_trim(dev.handle))
        if not args.serve_only_new:
            out[name]["phi3_same_size"] = phi3_leg(dev, torch, stream, c, peaks, args.steps)
        dev.check(dev._lib.rcu_pool_trim(dev.handle))
    last = out[sizes[-1]][models[0]]
    print(json.dumps({"metric": models[0] + "_decode_tokens_per_s", "value": last["decode_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": args.steps,
                      "warmup": 3, "ms_per_step": last["decode_us"] / 1e3, "higher_is_better": True, "dtype": "bf16", "data": "synthetic",
                      "peaks": {"hbm_gbs": peaks[0], "bf16_tflops": peaks[1], "bf16_tflops_sustained": peaks[2], "kind": "measured" if measured else "fallback"},
                      "clocks": sampler.stop(), "sizes": out}))
    dev.close()
