"""The Dadezen decoder end to end on the device - loader, lazy graph, fused decode step, engine, command line - against the
plain float64 restatement, on small random models of awkward sizes in both compute dtypes."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import dadezen_plain as dz

from . import dadezen_builders as B

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOKENS = 310
# root mean square of the logit error over that of the logits
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}


@pytest.fixture(scope="module")
def dev():
    from ratchet_b200 import Device
    d = Device(0)
    yield d
    d.close()


_cache = {}


def case(name, tmp_path_factory):
    """(folder, config, weights, tokens, float64 logits of every place) of a test model; computed once."""
    if name not in _cache:
        cfg = B.CONFIGS[name]
        W = B.weights(cfg, seed=sorted(B.CONFIGS).index(name) + 11)
        tokens = np.random.Generator(np.random.PCG64(7)).integers(0, cfg["vocab"], TOKENS).tolist()
        folder = B.write_model(str(tmp_path_factory.mktemp(name)), cfg, W)
        _cache[name] = (folder, cfg, W, tokens, dz.forward(cfg, W, tokens))
    return _cache[name]


def rel(got, want):
    d = got - want
    return float(np.sqrt((d * d).mean(-1) / (want * want).mean()).max())


def load(dev, folder, dtype):
    from ratchet_b200.models import load_model
    return load_model(folder, dev, dtype)


@pytest.fixture(params=sorted(B.CONFIGS))
def model_case(request, tmp_path_factory):
    return case(request.param, tmp_path_factory)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_decoding_and_portions_agree_with_the_restatement(dev, model_case, dtype):
    folder, cfg, W, tokens, want = model_case
    m = load(dev, folder, dtype)
    places = list(range(TOKENS))
    # the whole prompt, with the residual stream after every layer run
    streams, ref = [], []
    got = m.prefill(tokens, m.new_state(), places, streams)
    assert rel(got, want) < LIMIT[dtype]
    dz.forward(cfg, W, tokens, ref)
    assert len(streams) == len(ref)
    for s, r in zip(streams, ref):
        assert rel(s.to_numpy(), r) < LIMIT[dtype]
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
def test_slots_are_independent_and_reusable(dev, tmp_path_factory, dtype):
    folder, cfg, W, tokens, want = case("mixed", tmp_path_factory)
    from ratchet_b200 import RatchetCudaError
    from ratchet_b200.engine import Engine
    e = Engine(load(dev, folder, dtype), TOKENS, slots=2, portion=50)      # prompts longer than a portion are cut by the engine
    other = tokens[::-1]
    other_want = dz.forward(cfg, W, other[:120])
    # two sequences of unequal length, interleaved; the ended one's slot is taken over twice
    a = [e.step("a", tokens[:170], [169])[0]]
    b = [e.step("b", other[:3], [2])[0]]
    with pytest.raises(RatchetCudaError):
        e.step("c", tokens[:4])
    for i in range(30):
        a.append(e.step("a", [tokens[170 + i]], [0])[0])
        b.append(e.step("b", other[3 + 2 * i:5 + 2 * i], [1])[0])
    assert rel(np.array(a), want[169:200]) < LIMIT[dtype]
    assert rel(np.array(b), other_want[[2] + list(range(4, 64, 2))]) < LIMIT[dtype]
    e.end("b")
    for cuts in ([40, 1, 1, 78], [1, 1, 118]):
        at, rows = 0, []
        for n in cuts:
            rows.append(e.step("c", other[at:at + n], list(range(n))))
            at += n
        e.end("c")
        assert rel(np.concatenate(rows), other_want) < LIMIT[dtype]
    assert rel(e.step("a", tokens[200:], list(range(TOKENS - 200))), want[200:]) < LIMIT[dtype]
    with pytest.raises(RatchetCudaError):
        e.step("a", [1])                                                    # the slot is full
    with pytest.raises(RatchetCudaError):
        e.step("d", [cfg["vocab"]])


def greedy(cfg, W, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(dz.forward(cfg, W, seq)[-1])))
    return seq[len(prompt):]


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_scheduler(dev, tmp_path_factory, name):
    folder, cfg, W, tokens, _ = case(name, tmp_path_factory)
    from ratchet_b200.engine import Engine, Request, Sampler
    e = Engine(load(dev, folder, "float32"), 200, slots=2)
    prompts = [tokens[:45], tokens[60:61], tokens[100:138], tokens[5:9]]
    wants = [greedy(cfg, W, p, n) for p, n in zip(prompts, (12, 20, 3, 9))]
    done = e.run([Request(p, len(w)) for p, w in zip(prompts, wants)])
    assert [r.output for r in done] == wants
    assert e.generate(prompts[0], 12, stop=wants[0][4]) == wants[0][:wants[0].index(wants[0][4]) + 1]
    sampled = e.generate(prompts[0], 8, Sampler(temperature=0.8, top_k=5, seed=3))
    assert sampled == e.generate(prompts[0], 8, Sampler(temperature=0.8, top_k=5, seed=3)) and all(0 <= t < cfg["vocab"] for t in sampled)


def test_long_decoding_wraps_every_ring(dev, tmp_path_factory):
    """Hundreds of decoded tokens after a short prompt: the rings wrap many times and the states keep what they should."""
    folder, cfg, W, _, _ = case("odd", tmp_path_factory)
    tokens = np.random.Generator(np.random.PCG64(9)).integers(0, cfg["vocab"], 900).tolist()
    want = dz.forward(cfg, W, tokens)
    m = load(dev, folder, "float32")
    st = m.new_state()
    m.prefill(tokens[:4], st)
    got = np.concatenate([m.decode(st, t)[0].to_numpy() for t in tokens[4:]])
    assert rel(got, want[4:]) < LIMIT["float32"]


def test_decode_step_replays_one_graph_and_counts_its_kernels(dev, tmp_path_factory):
    folder, cfg, _, tokens, _ = case("plain", tmp_path_factory)
    m = load(dev, folder, "bfloat16")
    st = m.new_state()
    for t in tokens[:3]:
        m.decode(st, t)
    n = st.stack.kernels_per_step
    assert n == 3 + 3 + 6                   # embedding, head, arg-max; a lightning run; a latent run
    before = dev.launches
    m.decode(st)
    assert dev.launches == before + n
    dev.sync()


def test_trace_command(tmp_path, tmp_path_factory):
    folder, cfg, W, tokens, want = case("plain", tmp_path_factory)
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
    bad = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float16", "--out", str(tmp_path)], input="", capture_output=True)
    assert bad.returncode == 3


def test_generate_command(tmp_path_factory):
    folder, cfg, W, tokens, _ = case("plain", tmp_path_factory)
    p = subprocess.run([sys.executable, "-m", "ratchet_b200", "generate", "--model", folder, "--dtype", "float32", "--tokens",
                        ",".join(str(t) for t in tokens[:20]), "--max-new", "6"], capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [int(t) for t in p.stdout.split()] == greedy(cfg, W, tokens[:20], 6)
