"""The Mefesun decoder end to end on the device - loader, lazy graph, fused decode step, engine, command line - against the
plain float64 restatement, on small random models of awkward sizes in both compute dtypes."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import mefesun_plain as mp

from . import mefesun_builders as B
from .test_gpu_dadezen import LIMIT, dev, load, rel  # noqa: F401  (dev is a fixture)

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOKENS = 310

_cache = {}


def case(name, tmp_path_factory):
    """(folder, config, weights, tokens, float64 logits of every place, residual streams) of a test model; computed once."""
    if name not in _cache:
        cfg = B.CONFIGS[name]
        W = B.weights(cfg, seed=sorted(B.CONFIGS).index(name) + 21)
        tokens = np.random.Generator(np.random.PCG64(8)).integers(0, cfg["vocab"], TOKENS).tolist()
        streams = []
        want = mp.forward(cfg, W, tokens, streams)
        _cache[name] = (B.write_model(str(tmp_path_factory.mktemp(name)), cfg, W), cfg, W, tokens, want, streams)
    return _cache[name]


@pytest.fixture(params=sorted(B.CONFIGS))
def model_case(request, tmp_path_factory):
    return case(request.param, tmp_path_factory)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_decoding_and_portions_agree_with_the_restatement(dev, model_case, dtype):
    folder, cfg, W, tokens, want, ref = model_case
    m = load(dev, folder, dtype)
    # the whole prompt, with the residual stream after every layer run
    streams = []
    got = m.prefill(tokens, m.new_state(TOKENS), list(range(TOKENS)), streams)
    assert rel(got, want) < LIMIT[dtype]
    assert len(streams) == len(ref)
    for s, r in zip(streams, ref):
        assert rel(s.to_numpy()[:, :cfg["width"]], r) < LIMIT[dtype]
    # token by token from the start
    st = m.new_state(TOKENS)
    got = np.concatenate([m.decode(st, t)[0].to_numpy() for t in tokens])
    assert rel(got, want) < LIMIT[dtype]
    # portions of changing size, single tokens among them
    from ratchet_b200.engine import Engine
    e = Engine(m, TOKENS)
    for cuts in ([2] * 155, [64, 64, 2, 1, 1, 3, 129, 46], [1, 5, 128, 2, 37, 36, 38, 63], [200] + [1] * 110):
        at, rows = 0, []
        for n in cuts:
            rows.append(e.step("a", tokens[at:at + n], list(range(n))))
            at += n
        e.end("a")
        assert at == TOKENS and rel(np.concatenate(rows), want) < LIMIT[dtype], cuts[:4]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk,sizes", [(1, {}), (5, {}), (16, {}), (17, dict(heads=20, kv_heads=1)), (33, dict(dim=18, vdim=10)), (64, dict(dim=128, vdim=128)),
                                         (150, dict(heads=3, kv_heads=3, dim=72, vdim=8))])
def test_a_loud_token_is_seen_in_its_chunk_only(dev, tmp_path, dtype, chunk, sizes):
    """Loud tokens at a chunk's first and last places, seen or not by prompts, portions and decoded tokens on either side of the edge."""
    cfg, W = B.loud_case(chunk, **sizes)
    n = 4 * chunk + 3 if chunk > 1 else 12
    tokens = [2 + k % 30 for k in range(n)]
    for at in (0, 2 * chunk - 1, 2 * chunk):
        tokens[at] = 1
    want = mp.forward(cfg, W, tokens)
    m = load(dev, B.write_model(str(tmp_path), cfg, W), dtype)
    limit = LIMIT[dtype]
    assert rel(m.prefill(tokens, m.new_state(n), list(range(n))), want) < limit
    st = m.new_state(n)
    assert rel(np.concatenate([m.decode(st, t)[0].to_numpy() for t in tokens]), want) < limit
    for first in sorted({chunk, 2 * chunk - 1, 2 * chunk, 2 * chunk + 1} - {1}):
        st = m.new_state(n)
        got = [m.prefill(tokens[:first], st, list(range(first)))]
        got += [m.decode(st, t)[0].to_numpy() for t in tokens[first:first + 3]]
        rest = n - first - 3
        if rest > 1:
            got.append(m.prefill(tokens[first + 3:], st, list(range(rest))))
        got = np.concatenate(got)
        assert rel(got, want[:len(got)]) < limit, first


@pytest.mark.parametrize("sizes", [{}, dict(dim=128, vdim=64, heads=6), dict(dim=18, vdim=10)])
def test_caches_of_thousands_of_rows(dev, tmp_path, sizes):
    """The decode attention of a cache that more CTAs share than a cluster holds."""
    cfg, W = B.loud_case(6000, **sizes)
    tokens = [1 if k in (0, 130) else 2 + k % 30 for k in range(300)]
    want = mp.forward(cfg, W, tokens)
    m = load(dev, B.write_model(str(tmp_path), cfg, W), "bfloat16")
    st = m.new_state()
    got = [m.prefill(tokens[:100], st, list(range(100)))] + [m.decode(st, t)[0].to_numpy() for t in tokens[100:]]
    assert rel(np.concatenate(got), want) < LIMIT["bfloat16"]


def test_without_a_mask_every_position_is_seen(dev, tmp_path):
    cfg, W = B.loud_case(7)
    del cfg["layers"][0]["mixer"]["mask"]
    tokens = [1] + [2 + k % 30 for k in range(99)]
    want = mp.forward(cfg, W, tokens)
    m = load(dev, B.write_model(str(tmp_path), cfg, W), "float32")
    from ratchet_b200 import RatchetCudaError
    with pytest.raises(RatchetCudaError):
        m.new_state()                                        # such a layer's cache needs a length
    st = m.new_state(100)
    got = [m.prefill(tokens[:30], st, list(range(30))), m.prefill(tokens[30:50], st, list(range(20)))]
    got += [m.decode(st, t)[0].to_numpy() for t in tokens[50:]]
    assert rel(np.concatenate(got), want) < LIMIT["float32"]
    with pytest.raises(RatchetCudaError):
        m.decode(st, 3)                                      # full


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_are_independent_and_reusable(dev, tmp_path_factory, dtype):
    folder, cfg, W, tokens, want, _ = case("mixed", tmp_path_factory)
    from ratchet_b200 import RatchetCudaError
    from ratchet_b200.engine import Engine
    e = Engine(load(dev, folder, dtype), TOKENS, slots=2, portion=50)
    other = tokens[::-1]
    other_want = mp.forward(cfg, W, other[:120])
    a = [e.step("a", tokens[:170], [169])[0]]
    b = [e.step("b", other[:3], [2])[0]]
    for i in range(30):
        a.append(e.step("a", [tokens[170 + i]], [0])[0])
        b.append(e.step("b", other[3 + 2 * i:5 + 2 * i], [1])[0])
    assert rel(np.array(a), want[169:200]) < LIMIT[dtype]
    assert rel(np.array(b), other_want[[2] + list(range(4, 64, 2))]) < LIMIT[dtype]
    e.end("b")
    for cuts in ([40, 1, 1, 78], [1, 1, 118]):                # the ended sequence's slot, twice
        at, rows = 0, []
        for n in cuts:
            rows.append(e.step("c", other[at:at + n], list(range(n))))
            at += n
        e.end("c")
        assert rel(np.concatenate(rows), other_want) < LIMIT[dtype]
    assert rel(e.step("a", tokens[200:], list(range(TOKENS - 200))), want[200:]) < LIMIT[dtype]
    with pytest.raises(RatchetCudaError):
        e.step("a", [1])


def greedy(cfg, W, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(mp.forward(cfg, W, seq)[-1])))
    return seq[len(prompt):]


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_scheduler(dev, tmp_path_factory, name):
    folder, cfg, W, tokens, _, _ = case(name, tmp_path_factory)
    from ratchet_b200.engine import Engine, Request, Sampler
    e = Engine(load(dev, folder, "float32"), 200, slots=2)
    prompts = [tokens[:45], tokens[60:61], tokens[100:138], tokens[5:9]]
    wants = [greedy(cfg, W, p, n) for p, n in zip(prompts, (12, 14, 3, 9))]
    done = e.run([Request(p, len(w)) for p, w in zip(prompts, wants)])
    assert [r.output for r in done] == wants
    sampled = e.generate(prompts[0], 8, Sampler(temperature=0.8, top_k=5, seed=3))
    assert sampled == e.generate(prompts[0], 8, Sampler(temperature=0.8, top_k=5, seed=3)) and all(0 <= t < cfg["vocab"] for t in sampled)


def test_long_decoding_fills_and_leaves_many_chunks(dev, tmp_path_factory):
    folder, cfg, W, _, _, _ = case("odd", tmp_path_factory)
    tokens = np.random.Generator(np.random.PCG64(9)).integers(0, cfg["vocab"], 700).tolist()
    want = mp.forward(cfg, W, tokens)
    m = load(dev, folder, "float32")
    st = m.new_state()
    m.prefill(tokens[:4], st)
    got = np.concatenate([m.decode(st, t)[0].to_numpy() for t in tokens[4:]])
    assert rel(got, want[4:]) < LIMIT["float32"]


def test_decode_step_replays_one_graph_and_counts_its_kernels(dev, tmp_path_factory):
    folder, cfg, _, tokens, _, _ = case("mixed", tmp_path_factory)
    m = load(dev, folder, "bfloat16")
    st = m.new_state(TOKENS)
    for t in tokens[:3]:
        m.decode(st, t)
    n = st.stack.kernels_per_step
    assert n == 3 + 4 * 5 + 3               # embedding, head, arg-max; four layers with a feed-forward, one without
    before = dev.launches
    m.decode(st)
    assert dev.launches == before + n
    dev.sync()


def test_layers_that_share_weights_keep_caches_of_their_own(dev, tmp_path_factory):
    folder, cfg, _, _, _, _ = case("mixed", tmp_path_factory)
    m = load(dev, folder, "float32")
    assert [i for i, l in enumerate(m.graph.layers) if l is not None] == [0, 1, 3] and m.graph.order == [0, 1, 0, 3, 0]
    st = m.new_state(64)
    assert len({t.data_ptr() for t in st.runs}) == 5
    assert [t.shape()[0] for t in st.runs] == [37, 5, 37, 64, 37]


def test_trace_and_generate_commands(tmp_path, tmp_path_factory):
    folder, cfg, W, tokens, want, _ = case("many", tmp_path_factory)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:90], "want": [3, 89]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tokens[90:91], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": tokens[91:94], "want": [0, 1, 2]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": tokens[:1], "want": [0]}], "end": ["y"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "100"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert p.returncode == 0, p.stderr[-2000:]
        assert p.stdout.split() == "done 0 done 1 done 2 done 3".split()
        for k, rows in ((0, [3, 89]), (2, [91, 92, 93]), (3, [0])):
            got = np.fromfile(out / f"{k}.f32", "<f4").reshape(len(rows), -1)
            assert rel(got, want[rows]) < LIMIT[dtype]
        assert not (out / "1.f32").exists()
    p = subprocess.run([sys.executable, "-m", "ratchet_b200", "generate", "--model", folder, "--dtype", "float32", "--tokens",
                        ",".join(str(t) for t in tokens[:20]), "--max-new", "6"], capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [int(t) for t in p.stdout.split()] == greedy(cfg, W, tokens[:20], 6)
