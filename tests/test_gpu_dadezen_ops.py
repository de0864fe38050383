"""Each mechanism of the Dadezen decoder through the device ABI against the plain float64 restatement (oracle/dadezen_plain.py)
or numpy, alone: sizes with and without the kernels' alignment, both compute dtypes, state and ring carried over portions."""
import numpy as np
import pytest

from oracle import dadezen_plain as dz
from ratchet_b200 import capi

pytestmark = pytest.mark.gpu

F32, BF16, F16 = capi.F32, capi.BF16, capi.F16


@pytest.fixture(scope="module")
def dev():
    from ratchet_b200 import Device
    d = Device(0)
    yield d
    d.close()


def rng(seed):
    return np.random.Generator(np.random.PCG64(seed))


def put(dev, a, dt):
    """Device buffer and the values it really holds."""
    a = np.asarray(a, np.float32)
    if dt == BF16:
        u = capi.to_bf16(a)
        return dev.from_numpy(u, dt=BF16), capi.from_bf16(u).astype(np.float64)
    if dt == F16:
        return dev.from_numpy(a.astype(np.float16)), a.astype(np.float16).astype(np.float64)
    return dev.from_numpy(a), a.astype(np.float64)


def get(buf):
    a = buf.to_numpy()
    return capi.from_bf16(a) if buf.dt == BF16 else a.astype(np.float32)


def err(got, want):
    return float(np.abs(got - want).max() / max(np.abs(want).max(), 1e-30))


TOL = {F32: 3e-6, BF16: 6e-3, F16: 1e-3}


def test_bf16_conversion_helpers():
    x = np.array([1.0, -2.5, 3.1415927, 1e-40, 65504.0, np.inf, 0.0], np.float32)
    import torch
    assert np.array_equal(capi.to_bf16(x), torch.from_numpy(x).bfloat16().view(torch.int16).numpy().view(np.uint16))


# ---------------------------------------------------------------------------------------- Linear
@pytest.mark.parametrize("dt", [F32, BF16, F16])
@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (3, 33, 45), (4, 200, 264), (5, 33, 45), (2, 64, 64), (37, 128, 192), (64, 72, 80), (129, 264, 328),
                                   (300, 520, 1096), (700, 1024, 512)])
def test_linear_output_types_and_epilogue(dev, dt, M, N, K):
    g = rng(M * 1000 + N)
    w, wv = put(dev, g.standard_normal((N, K)) / np.sqrt(K), dt)
    x, xv = put(dev, g.standard_normal((M, K + 24)), dt)
    for col in (0, 8):
        want = xv[:, col:col + K] @ wv.T
        assert err(get(dev.linear(w, x, x_col=col, dt=dt)), want) < TOL[dt]
        assert err(get(dev.linear(w, x, x_col=col, dt=F32)), want) < 3e-6
    b, bv = put(dev, g.standard_normal(N), F32)
    r, rv = put(dev, 4 * g.standard_normal((M, N)), F32)
    z = xv[:, :K] @ wv.T + bv
    n = N // 2
    z[:, :n] = dz.silu(z[:, :n])
    out = dev.linear(w, x, bias=b, resid=r, alpha=0.3, act="silu", act_cols=n, dt=F32)
    assert err(get(out), rv + 0.3 * z) < 3e-6
    dev.linear(w, x, bias=b, resid=r, alpha=0.3, act="silu", act_cols=n, dt=F32, out=r)          # into the residual itself
    assert np.array_equal(get(r), get(out))


def test_linear_refuses_what_it_cannot_do(dev):
    from ratchet_b200 import RatchetCudaError
    w, _ = put(dev, np.ones((8, 8)), BF16)
    x, _ = put(dev, np.ones((2, 8)), BF16)
    r, _ = put(dev, np.ones((2, 8)), F32)
    for bad in (lambda: dev.linear(w, x, x_col=1), lambda: dev.linear(w, x, resid=r), lambda: dev.linear(w, r), lambda: dev.linear(w, x, act="silu", act_cols=9)):
        with pytest.raises(RatchetCudaError):
            bad()


# ---------------------------------------------------------------------------------------- row operations
@pytest.mark.parametrize("out", [F32, BF16, F16])
@pytest.mark.parametrize("rows,N", [(1, 1), (5, 33), (3, 128), (9, 130), (7, 512), (6, 700), (3, 3000)])
def test_norms_with_column_windows_and_gates(dev, out, rows, N):
    g = rng(rows + N)
    x, xv = put(dev, 50.0 + g.standard_normal((rows, N + 11)), F32)      # a mean far above the deviations
    s, sv = put(dev, g.standard_normal(N), F32)
    gate, gv = put(dev, 2 * g.standard_normal((rows, N + 5)), out)
    for col in (0, 7):
        win = xv[:, col:col + N]
        assert err(get(dev.norm_rows(capi.LAYER_NORM, x, s, 1e-5, out, col=col)), dz.layer_norm(win, sv, 1e-5)) < max(TOL[out], 3e-5)
        want = dz.rms_norm(win, sv, 1e-3)
        assert err(get(dev.norm_rows(capi.RMS_NORM, x, s, 1e-3, out, col=col)), want) < TOL[out]
        assert err(get(dev.norm_rows(capi.RMS_NORM, x, s, 1e-3, out, col=col, gate=gate, gate_col=5)), want * dz.sigmoid(gv[:, 5:])) < TOL[out]


@pytest.mark.parametrize("dt", [F32, BF16, F16])
@pytest.mark.parametrize("rows,F", [(1, 1), (3, 17), (5, 64), (40, 1000)])
def test_gated_activation(dev, dt, rows, F):
    x, xv = put(dev, 3 * rng(F).standard_normal((rows, 2 * F)), dt)
    for name, fn in (("gelu", dz.gelu_tanh), ("silu", dz.silu)):
        assert err(get(dev.glu(name, x)), fn(xv[:, :F]) * xv[:, F:]) < TOL[dt]


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("rot", [{"dims": 8, "base": 10000.0}, {"dims": 6, "base": 500.0, "scaling": {"factor": 8.0, "original": 128, "fast": 8.0, "slow": 1.0}},
                                 {"dims": 64, "base": 50000.0, "scaling": {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}}])
def test_rotation_at_near_and_far_positions(dev, dt, rot):
    s = rot.get("scaling")
    table, mag = capi.rotary_frequencies(rot["dims"], rot["base"], *([s[k] for k in ("factor", "original", "fast", "slow")] if s else []))
    f, m = dz.rotary_frequencies(rot)
    assert np.allclose(table.astype(np.float64).sum(0), f, rtol=1e-13) and abs(mag - m) < 1e-7
    fr, _ = put(dev, table, F32)
    for pos in (0, 3, 131071):
        x, xv = put(dev, rng(pos).standard_normal((5, 3, rot["dims"] + 9)), dt)
        want = xv.copy()
        want[..., 4:4 + rot["dims"]] = dz.rotate(xv[..., 4:4 + rot["dims"]], np.arange(pos, pos + 5), rot)
        got = dev.rotary(x, fr, mag, pos, first=4)
        assert err(get(got), want) < (1e-6 if dt == F32 else TOL[dt])
        dev.rotary(x, fr, mag, pos, first=4, out=x)
        assert np.array_equal(get(x), get(got))


# ---------------------------------------------------------------------------------------- linear attention
def powers(decay, n=129):
    return np.power(np.asarray(decay, np.float64)[:, None], np.arange(n)[None])


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,D,E,decay", [(1, 1, 1, (0.5,)), (3, 24, 40, (0.02, 0.9, 0.999)), (2, 9, 13, (1.0, 0.97)), (2, 64, 64, (0.6, 0.99)),
                                         (2, 128, 128, (0.93, 0.9995)), (1, 200, 72, (0.98,)), (1, 300, 20, (0.9,)), (2, 32, 136, (0.0, 0.9))])
def test_linear_attention_in_portions(dev, dt, H, D, E, decay):
    g = rng(H * D + E)
    T = 300
    x = g.standard_normal((T, 2 * H * D + H * E + 8)) * 0.5
    x[40, H * D:2 * H * D] *= 30.0          # one key that stands out for hundreds of tokens
    _, xv = put(dev, x, dt)
    q, k, v = xv[:, :H * D].reshape(T, H, D), xv[:, H * D:2 * H * D].reshape(T, H, D), xv[:, 2 * H * D:2 * H * D + H * E].reshape(T, H, E)
    want, S = dz.linear_attention(q, k, v, np.float32(decay).astype(np.float64))
    dp, _ = put(dev, powers(decay), F32)
    for cut in ([T], [2, 2, 296], [127, 1, 128, 44], [33, 64, 3, 200], [255, 45]):
        state = dev.zeros(F32, (H, D, E))
        at, out = 0, []
        for n in cut:
            b, _ = put(dev, x[at:at + n], dt)
            out.append(get(dev.lightning(b, dp, state)))
            at += n
        out = np.concatenate(out).reshape(T, H, E)
        for t in (0, 1, 41, 127, 128, 129, T - 1):          # at every scale: the outputs differ by orders of magnitude
            assert err(out[t], want[t]) < (5e-5 if dt == BF16 else 2e-5), (cut, t)
        assert err(state.to_numpy(), S) < (5e-5 if dt == BF16 else 5e-6), cut


# ---------------------------------------------------------------------------------------- latent attention
def latent_case(g, T, H, D, R, E, C):
    return (g.standard_normal((T, H, D + R)), g.standard_normal((T, 3 + C + R)), 1 + 0.1 * g.standard_normal(C),
            g.standard_normal((H * D, C)) / np.sqrt(C), g.standard_normal((H * E, C)) / np.sqrt(C))


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,D,R,E,C,window", [(1, 8, 2, 9, 12, 1), (3, 5, 6, 7, 21, 11), (2, 16, 8, 24, 64, 64), (2, 32, 32, 32, 96, 65), (4, 64, 32, 64, 128, 100),
                                              (1, 128, 64, 128, 144, 1000), (2, 24, 8, 144, 40, 129), (1, 16, 16, 300, 32, 50)])
def test_latent_ring_and_window(dev, dt, H, D, R, E, C, window):
    g = rng(window)
    T = 280
    q, low, scale, uk, uv = latent_case(g, T, H, D, R, E, C)
    rot = {"dims": R, "base": 1000.0, "scaling": {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}}
    table, mag = capi.rotary_frequencies(R, 1000.0, 4.0, 32, 8.0, 1.0)
    fr, _ = put(dev, table, F32)
    sc, scv = put(dev, scale, F32)
    wkv, wv = put(dev, np.concatenate([uk, uv]), dt)
    _, qv = put(dev, q, dt)
    _, lowv = put(dev, low, F32)
    rnd = (lambda a: capi.from_bf16(capi.to_bf16(a.astype(np.float32))).astype(np.float64)) if dt == BF16 else (lambda a: a)
    c = rnd(dz.rms_norm(lowv[:, 3:3 + C], scv, 1e-5))
    kr = rnd(dz.rotate(lowv[:, 3 + C:], np.arange(T), rot))
    k = np.concatenate([rnd(c @ wv[:H * D].T).reshape(T, H, D), np.repeat(kr[:, None], H, 1)], -1)
    v = rnd(c @ wv[H * D:].T).reshape(T, H, E)
    want = dz.windowed_softmax_attention(qv, k, v, 0.4, window).reshape(T, H * E)
    for cut in ([T], [2, 3, 275], [1, 64, 1, 128, 86], [window % 97 + 2, 130, T - 132 - window % 97]):
        ring = dev.zeros(dt, (min(window, T), C + R))
        at, out = 0, []
        for n in cut:
            lb, _ = put(dev, low[at:at + n], F32)
            qb, _ = put(dev, q[at:at + n], dt)
            seen = dev.latent_append(lb, sc, 1e-5, fr, mag, at, ring, n + min(at, window - 1), col=3)
            out.append(get(dev.window_attention(qb, dev.linear(wkv, seen, dt=dt), seen, C, E, window, 0.4)))
            at += n
        assert err(np.concatenate(out), want) < (1e-2 if dt == BF16 else 5e-6), cut


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 63, 64, 65, 127, 128, 129, 200])
def test_window_edges_show_a_single_loud_key(dev, dt, window):
    """One key scores far above all others and its value is unique: queries up to window - 1 rows later return that value, the
    query `window` rows later does not."""
    T, H, D, R, E, at = 640, 2, 16, 8, 16, 350
    g = rng(window)
    q = np.abs(g.standard_normal((T, H, D + R))) + 0.5
    k = 0.05 * g.standard_normal((T, H * D + H * E))
    k[:, H * D:] = g.standard_normal((T, H * E))
    k[at, :H * D] = 4.0
    k[at, H * D:] = 50.0
    sh = 0.05 * g.standard_normal((T, R))
    for t0, n in ((0, T), (at, 250), (at + window - 1, 2), (at + window, 3), (at + max(window - 2, 0), 40)):
        lo = max(0, t0 - window + 1)
        qb, qv = put(dev, q[t0:t0 + n], dt)
        kb, kv = put(dev, k[lo:t0 + n], dt)
        sb, sv = put(dev, sh[lo:t0 + n], dt)
        got = get(dev.window_attention(qb, kb, sb, 0, E, window, 1.0)).reshape(n, H, E)
        full_k = np.concatenate([kv[:, :H * D].reshape(-1, H, D), np.repeat(sv[:, None], H, 1)], -1)
        full_q = np.zeros((len(kv), H, D + R))
        full_q[-n:] = qv
        want = dz.windowed_softmax_attention(full_q, full_k, kv[:, H * D:].reshape(-1, H, E), 1.0, window)[-n:]
        assert np.abs(got - want).max() < (0.3 if dt == BF16 else 1e-3)
        for t in range(t0, t0 + n):
            assert (got[t - t0].min() > 40) == (at <= t < at + window), t
