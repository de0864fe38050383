"""Each mechanism of the Mefesun decoder through the device ABI, alone, against the plain float64 restatement (oracle/mefesun_plain.py)
or numpy: sizes with and without the kernels' alignment, both compute dtypes, rings carried over portions."""
import numpy as np
import pytest

from oracle import dadezen_plain as dz
from oracle import mefesun_plain as mp
from ratchet_b200 import capi

from .test_gpu_dadezen_ops import BF16, F32, TOL, dev, err, get, put, rng  # noqa: F401  (dev is a fixture)

pytestmark = pytest.mark.gpu

YARN = {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}


def round_to(a, dt):
    return capi.from_bf16(capi.to_bf16(np.asarray(a, np.float32))).astype(np.float64) if dt == BF16 else np.asarray(a, np.float64)


# ---------------------------------------------------------------------------------------- products and norms
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("M,N,K", [(1, 40, 64), (3, 33, 45), (40, 72, 80), (300, 520, 328)])
def test_linear_activations(dev, dt, M, N, K):
    g = rng(M + N)
    w, wv = put(dev, g.standard_normal((N, K)) / np.sqrt(K), dt)
    x, xv = put(dev, 2 * g.standard_normal((M, K + 8)), dt)
    z = xv[:, 8:] @ wv.T
    for out in (dt, F32):
        b, bv = put(dev, g.standard_normal(N), out)
        assert err(get(dev.linear(w, x, bias=b, x_col=8, act="relu_squared", dt=out)), mp.squared_relu(z + bv)) < max(TOL[out], 3e-6)
        want = z + bv
        want[:, :N // 3] = mp.softcap(want[:, :N // 3], 1.5)
        assert err(get(dev.linear(w, x, bias=b, x_col=8, act="softcap", act_cols=N // 3, act_param=1.5, dt=out)), want) < max(TOL[out], 3e-6)


def test_linear_refuses_unknown_activations(dev):
    from ratchet_b200 import RatchetCudaError
    w, _ = put(dev, np.ones((8, 8)), BF16)
    x, _ = put(dev, np.ones((2, 8)), BF16)
    with pytest.raises(RatchetCudaError):
        dev.linear(w, x, act="softcap", act_param=0.0)
    with pytest.raises(KeyError):
        dev.linear(w, x, act="other")


@pytest.mark.parametrize("out", [F32, BF16])
@pytest.mark.parametrize("rows,N", [(1, 1), (5, 33), (9, 130), (6, 700), (3, 3000)])
def test_norms_with_a_shift(dev, out, rows, N):
    g = rng(rows + N)
    x, xv = put(dev, 5.0 + g.standard_normal((rows, N + 4)), F32)
    s, sv = put(dev, g.standard_normal(N), F32)
    b, bv = put(dev, g.standard_normal(N), F32)
    for col in (0, 4):
        got = get(dev.norm_rows(capi.LAYER_NORM, x, s, 1e-2, out, col=col, shift=b))
        assert err(got, mp.layer_norm_bias(xv[:, col:col + N], sv, bv, 1e-2)) < max(TOL[out], 3e-5)


@pytest.mark.parametrize("copy", [F32, BF16])
@pytest.mark.parametrize("rows,W", [(1, 1), (4, 45), (3, 80), (7, 1024), (2, 1032), (3, 3000), (2, 8192), (1, 9000)])
def test_stream_rows_and_post_norm(dev, copy, rows, W):
    g = rng(W)
    x, xv = put(dev, g.standard_normal((rows, W)), BF16)
    y, yv = put(dev, 3.0 + 2 * g.standard_normal((rows, W)), F32)
    s, sv = put(dev, g.standard_normal(W), F32)
    b, bv = put(dev, g.standard_normal(W), F32)

    def parts(buf):
        a = buf.to_numpy()
        tail = capi.from_bf16(np.ascontiguousarray(a[:, W:]).view(np.uint16)[:, :W]) if copy == BF16 else None
        assert a.shape[1] == (W + (W + 1) // 2 if copy == BF16 else W)
        return a[:, :W], tail

    st = dev.stream_rows(x, copy)
    v, c = parts(st)
    assert np.array_equal(v, xv) and (c is None or np.array_equal(c, xv))
    want = xv + mp.layer_norm_bias(yv, sv, bv, 1e-3)
    new = dev.post_norm(st, y, s, b, 1e-3)
    v, c = parts(new)
    assert err(v, want) < 3e-6
    assert c is None or np.array_equal(c, capi.from_bf16(capi.to_bf16(v)))
    dev.post_norm(st, y, s, b, 1e-3, out=st)                    # in place
    assert np.array_equal(st.to_numpy()[:, :W], v)


# ---------------------------------------------------------------------------------------- heads
def angle_table(dev, rot, pos, n):
    s = rot.get("scaling")
    table, mag = capi.rotary_frequencies(rot["dims"], rot["base"], *([s[k] for k in ("factor", "original", "fast", "slow")] if s else []))
    fr, _ = put(dev, table, F32)
    return dev.rotary_angles(fr, mag, pos, n)


def test_rotary_angles_near_and_far(dev):
    rot = {"dims": 12, "base": 500.0, "scaling": YARN}
    f, m = dz.rotary_frequencies(rot)
    for pos in (0, 7, 131071):
        a = angle_table(dev, rot, pos, 5).to_numpy().reshape(5, 6, 2)
        t = np.arange(pos, pos + 5)[:, None] * f[None]
        assert np.abs(a[..., 0] - m * np.cos(t)).max() < 3e-7 and np.abs(a[..., 1] - m * np.sin(t)).max() < 3e-7


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("T,H,D,dims", [(1, 1, 2, 2), (5, 3, 9, 4), (6, 2, 24, 8), (6, 7, 24, 6), (9, 5, 64, 14), (33, 4, 64, 64), (7, 5, 128, 96), (3, 2, 256, 64), (4, 1, 300, 128)])
def test_head_norm_and_rotation(dev, dt, T, H, D, dims):
    g = rng(D)
    rot = {"dims": dims, "base": 1000.0, "scaling": YARN}
    s, sv = put(dev, 1 + 0.5 * g.standard_normal(D), F32)
    for pos, col in ((0, 0), (1000, 8), (77, 3)):
        x, xv = put(dev, g.standard_normal((T, col + H * D + 8)), dt)
        want = dz.rotate(dz.rms_norm(xv[:, col:col + H * D].reshape(T, H, D), sv, 1e-2), np.arange(pos, pos + T), rot)
        got = get(dev.norm_rotary(x, H, s, 1e-2, angle_table(dev, rot, pos, T), col=col))
        assert got.shape == (T, H, D) and err(got, want) < max(TOL[dt], 3e-6)


SHAPES = [(1, 1, 8, 8, 1), (3, 1, 5, 7, 11), (6, 2, 24, 40, 37), (4, 4, 64, 64, 64), (8, 2, 128, 128, 100), (20, 1, 32, 32, 130), (2, 2, 200, 136, 48),
          (2, 1, 16, 300, 1000), (4, 2, 48, 72, 257), (6, 3, 40, 24, None)]


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,G,D,E,chunk", SHAPES)
def test_ring_and_chunks_in_portions(dev, dt, H, G, D, E, chunk):
    g = rng(D * E)
    T, dims = 300, D // 4 * 2
    rot = {"dims": dims, "base": 1000.0, "scaling": YARN}
    scale, sink = 1.5 / np.sqrt(D), 2.0 * g.standard_normal(H)
    x = g.standard_normal((T, 3 + H * D + G * (D + E)))
    _, xv = put(dev, x, dt)
    qs, qsv = put(dev, 1 + 0.2 * g.standard_normal(D), F32)
    ks, ksv = put(dev, 1 + 0.2 * g.standard_normal(D), F32)
    sk, skv = put(dev, sink, F32)
    pos = np.arange(T)
    heads = lambda a, n, w: round_to(dz.rotate(dz.rms_norm(a.reshape(T, n, D), w, 1e-5), pos, rot), dt)
    q, k = heads(xv[:, 3:3 + H * D], H, qsv), heads(xv[:, 3 + H * D:3 + (H + G) * D], G, ksv)
    v = xv[:, 3 + (H + G) * D:].reshape(T, G, E)
    want = mp.sink_attention(q, k, v, scale, skv, chunk).reshape(T, H * E)
    seen = lambda p: p % chunk if chunk else p
    for cut in ([T], [2, 3, 295], [1, 64, 1, 128, 106], [36, 2, 1, 260, 1], [257, 43]):
        ring = dev.zeros(dt, (min(chunk or T, T), G * (D + E)))
        at, out = 0, []
        for n in cut:
            b, _ = put(dev, x[at:at + n], dt)
            an, old = angle_table(dev, rot, at, n), seen(at)
            qb = dev.norm_rotary(b, H, qs, 1e-5, an, col=3)
            kv = dev.kv_append(b, G, ks, 1e-5, an, at, min(n, seen(at + n)), ring, old + n, col=3 + H * D)
            out.append(get(dev.grouped_attention(qb, kv, G, E, scale, sk, chunk=chunk or 0, position=at - old)))
            at += n
        assert err(np.concatenate(out), want) < (1e-2 if dt == BF16 else 5e-6), cut


def test_ring_rows_are_positions_modulo_its_size(dev):
    """A block longer than the ring keeps its last rows; a block whose rows replace older ones still sees those."""
    G, D, E, R = 2, 8, 16, 10
    x = rng(1).standard_normal((40, G * (D + E)))
    s, sv = put(dev, np.ones(D), F32)
    _, xv = put(dev, x, BF16)
    rot = {"dims": 4, "base": 100.0}
    k = dz.rotate(dz.rms_norm(xv[:, :G * D].reshape(40, G, D), sv, 1e-5), np.arange(40), rot).reshape(40, G * D)
    rows = np.concatenate([k, xv[:, G * D:]], 1)
    ring = dev.zeros(BF16, (R, G * (D + E)))
    at = 0
    for n, old in ((25, 0), (3, 9), (12, 5)):
        b, _ = put(dev, x[at:at + n], BF16)
        keep = min(n, R)
        seen = get(dev.kv_append(b, G, s, 1e-5, angle_table(dev, rot, at, n), at, keep, ring, old + n))
        assert err(seen, rows[at - old:at + n]) < TOL[BF16]
        at += n
        held = get(ring)
        for p in range(at - R, at):
            assert err(held[p % R], rows[p]) < TOL[BF16]


def loud_block(g, T, H, G, D, E, at):
    """Queries and keys where one position's key scores far above all others and its value is unique."""
    q = np.abs(g.standard_normal((T, H, D))) + 0.5
    kv = 0.05 * g.standard_normal((T, G * (D + E)))
    kv[:, G * D:] = g.standard_normal((T, G * E))
    kv[at, :G * D] = 4.0
    kv[at, G * D:] = 50.0
    return q, kv


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("chunk", [1, 2, 16, 17, 63, 64, 65, 127, 128, 129, 200, 256])
def test_chunk_edges_show_a_single_loud_key(dev, dt, chunk):
    """Queries of the loud position's own chunk from it on return its value, all others do not - in whole blocks and in blocks that
    start anywhere in a chunk."""
    T, H, G, D, E = 640, 4, 2, 24, 16
    g = rng(chunk)
    for at in (350 // chunk * chunk, 350 // chunk * chunk + chunk - 1, 350):         # a chunk's first and last place, and some other
        q, kv = loud_block(g, T, H, G, D, E, at)
        for t0, n in ((0, T), (at, T - at), (at + 1, 2), (at // chunk * chunk + chunk - 1, 3), (at // chunk * chunk, chunk + 2)):
            lo = t0 // chunk * chunk
            qb, qv = put(dev, q[t0:t0 + n], dt)
            kb, kvv = put(dev, kv[lo:t0 + n], dt)
            got = get(dev.grouped_attention(qb, kb, G, E, 1.0, chunk=chunk, position=lo)).reshape(n, H, E)
            for t in range(t0, t0 + n):
                assert (got[t - t0].min() > 40) == mp.same_chunk(t, at, chunk), (at, t0, t)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("T", [3, 100, 300])
def test_windows_and_no_mask_of_grouped_heads(dev, dt, T):
    H, G, D, E, at = 4, 1, 32, 24, 1
    q, kv = loud_block(rng(T), T, H, G, D, E, at)
    qb, _ = put(dev, q, dt)
    kb, _ = put(dev, kv, dt)
    for window in (0, 1, 2, 70):
        got = get(dev.grouped_attention(qb, kb, G, E, 1.0, window=window)).reshape(T, H, E)
        for t in range(T):
            assert (got[t].min() > 40) == (at <= t and (window == 0 or t < at + window)), t


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("T", [4, 100, 300])
def test_sinks_take_their_share_once(dev, dt, T):
    """Equal scores: the output is the mean value times n / (n + exp(sink - score)), whatever the chunk's fill."""
    H, G, D, E, chunk = 4, 2, 16, 8, 40
    q, kv = np.ones((T, H, D)), np.ones((T, G * (D + E)))
    sink = np.array([-60.0, 4.0, 5.0, 90.0])
    qb, _ = put(dev, q, dt)
    kb, _ = put(dev, kv, dt)
    sk, _ = put(dev, sink, F32)
    got = get(dev.grouped_attention(qb, kb, G, E, 0.25, sk, chunk=chunk)).reshape(T, H, E)
    n = np.arange(T) % chunk + 1.0
    want = n[:, None] / (n[:, None] + np.exp(sink - 4.0))
    assert np.abs(got - want[..., None]).max() < (5e-3 if dt == BF16 else 2e-6)


def test_bad_arguments_are_refused(dev):
    from ratchet_b200 import RatchetCudaError
    q, _ = put(dev, np.ones((4, 3, 8)), BF16)
    kv, _ = put(dev, np.ones((4, 2 * 16)), BF16)
    s, _ = put(dev, np.ones(8), F32)
    x, _ = put(dev, np.ones((4, 32)), BF16)
    an = angle_table(dev, {"dims": 4, "base": 10.0}, 0, 4)
    ring = dev.zeros(BF16, (3, 32))
    sk, _ = put(dev, np.ones(2), F32)
    q4, _ = put(dev, np.ones((4, 4, 8)), BF16)
    for bad in (lambda: dev.grouped_attention(q, kv, 2, 8, 1.0), lambda: dev.grouped_attention(q4, kv, 2, 8, 1.0, sk),
                lambda: dev.kv_append(x, 2, s, 1e-5, an, 0, 4, ring, 4), lambda: dev.kv_append(x, 2, s, 1e-5, an, 9, 0, ring, 8),
                lambda: dev.kv_append(x, 2, s, 1e-5, an, 0, 0, ring, 4, col=1), lambda: dev.norm_rotary(x, 5, s, 1e-5, an)):
        with pytest.raises(RatchetCudaError):
            bad()
