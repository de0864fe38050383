"""Host side of the Dadezen decoder without a GPU: configuration, weight files, rotary tables, graph building, sequence slots,
scheduling and sampling; and the plain restatement's own consistency."""
import json

import numpy as np
import pytest

from oracle import dadezen_plain as dz
from ratchet_b200 import RatchetCudaError, capi
from ratchet_b200.engine import Engine, Request, Sampler
from ratchet_b200.models import REGISTRY, DadezenConfig, LatentConfig, LightningConfig, load_model
from ratchet_b200.nn import SequenceState
from ratchet_b200.safetensors import SafetensorsFile

from . import dadezen_builders as B


# ---------------------------------------------------------------------------------------- configuration
def test_configuration_is_read_and_ordered():
    for cfg in B.CONFIGS.values():
        c = DadezenConfig.read(json.loads(json.dumps(cfg)))
        assert c.runs() == dz.layer_order(cfg)
        for lc, e in zip(c.layers, cfg["layers"]):
            assert isinstance(lc.mixer, LightningConfig if e["type"] == "lightning" else LatentConfig)
            assert lc.mlp == bool(e["mlp"])
    c = DadezenConfig.read(B.CONFIGS["mixed"])
    assert c.runs() == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None)]
    assert c.layers[1].mixer.rot.factor == B.YARN["factor"] and c.layers[2].mixer.rot.factor == 0.0


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mixer"].update(decay=[0.5]),
                                    lambda c: c["layers"][0]["mlp"].update(kind="routed")])
def test_configurations_of_other_designs_are_refused(change):
    cfg = json.loads(json.dumps(B.CONFIGS["mixed"]))
    change(cfg)
    with pytest.raises(RatchetCudaError):
        DadezenConfig.read(cfg)
    bad = json.loads(json.dumps(B.CONFIGS["mixed"]))
    bad["loop"]["stop"] = 9
    with pytest.raises(RatchetCudaError):
        DadezenConfig.read(bad).runs()


def test_registry_names_the_class_by_architecture(tmp_path):
    assert "Dadezen" in REGISTRY
    (tmp_path / "config.json").write_text('{"architecture": "Nothing"}')
    with pytest.raises(RatchetCudaError, match="Nothing"):
        load_model(str(tmp_path), None)


# ---------------------------------------------------------------------------------------- files
def test_safetensors_reader(tmp_path):
    p = str(tmp_path / "t.safetensors")
    a = np.arange(12, dtype=np.float32).reshape(3, 4)
    i = np.array([[5, -6]], np.int32)
    B.write_safetensors(p, {"a": ("F32", a), "b": ("BF16", capi.to_bf16(a)), "i": ("I32", i)})
    f = SafetensorsFile(p)
    assert f.shape("b") == (3, 4) and "a" in f and "c" not in f
    assert np.array_equal(f.f32("a"), a) and np.array_equal(f.f32("b"), a) and np.array_equal(f.raw("i")[1], i)
    with pytest.raises(RatchetCudaError):
        f.raw("c")
    blob = open(p, "rb").read()
    n = int.from_bytes(blob[:8], "little")
    cases = {"short": blob[:-1], "header": (10 ** 9).to_bytes(8, "little") + blob[8:], "tiny": b"abc",
             "range": blob[:8] + blob[8:8 + n].replace(b"[0, 48]", b"[0, 40]") + blob[8 + n:]}
    for name, data in cases.items():
        q = tmp_path / name
        q.write_bytes(data)
        with pytest.raises(RatchetCudaError):
            SafetensorsFile(str(q))


def test_bf16_rounding_on_the_host():
    x = np.array([1.0, 1.00390625, 1.01171875, -3.0e38, 3.4e38, np.nan, np.inf, 1e-45], np.float32)
    got = capi.from_bf16(capi.to_bf16(x))
    assert got[1] == 1.0 and got[2] == np.float32(1.015625)          # ties go to the even mantissa
    assert np.isnan(got[5]) and np.isinf(got[6]) and np.isinf(got[4]) and got[3] < -2.9e38


@pytest.mark.parametrize("dims,base,sc", [(2, 10.0, None), (8, 10000.0, None), (6, 500.0, (4.0, 64, 16.0, 1.0)), (64, 50000.0, (40.0, 4096, 32.0, 1.0)),
                                          (16, 100.0, (2.0, 8, 32.0, 30.0)), (10, 1e6, (16.0, 1 << 20, 64.0, 0.25))])
def test_rotary_tables(dims, base, sc):
    rot = {"dims": dims, "base": base}
    if sc:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), sc))
    f, m = dz.rotary_frequencies(rot)
    table, mag = capi.rotary_frequencies(dims, base, *(sc or ()))
    assert np.allclose(table.astype(np.float64).sum(0), f, rtol=1e-13, atol=0) and abs(mag - m) < 1e-6
    with pytest.raises(RatchetCudaError):
        capi.rotary_frequencies(dims + 1, base)


# ---------------------------------------------------------------------------------------- slots, scheduling, sampling
class CountingModel:
    """A stand-in with the served-model interface: the logits name the position and the sum of the tokens seen."""
    vocab = 50

    def __init__(self):
        self.calls = []

    def new_state(self, max_tokens=None):
        s = SequenceState([])
        s.sum = 0
        return s

    def _one(self, st, token):
        if st.position == 0:
            st.sum = 0
        st.sum += token
        st.position += 1
        z = np.zeros(self.vocab, np.float32)
        z[(st.sum + st.position) % self.vocab] = 9.0
        return z

    def prefill(self, tokens, st, want=(), streams=None):
        self.calls.append(len(tokens))
        rows = [self._one(st, t) for t in tokens]
        return np.array([rows[w] for w in want], np.float32).reshape(len(want), self.vocab)

    def decode(self, st, token=None):
        self.calls.append(1)
        z = self._one(st, token)

        class Buf:
            def __init__(self, a):
                self.a = a

            def to_numpy(self):
                return self.a
        return Buf(z[None]), Buf(np.array([int(z.argmax())], np.int32))


def expected(prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append((sum(seq) + len(seq)) % 50)
    return seq[len(prompt):]


def test_steps_are_cut_into_portions_and_slots_are_reset():
    m = CountingModel()
    e = Engine(m, max_tokens=40, slots=1, portion=8)
    tokens = list(range(1, 18))
    got = e.step("a", tokens, [0, 7, 8, 16])
    assert m.calls == [8, 8, 1] and e.position("a") == 17
    assert [int(g.argmax()) for g in got] == [(sum(tokens[:k + 1]) + k + 1) % 50 for k in (0, 7, 8, 16)]
    with pytest.raises(RatchetCudaError):
        e.step("b", [1])                               # no slot
    for bad in ([50], [-1]):
        with pytest.raises(RatchetCudaError):
            e.step("a", bad)
    with pytest.raises(RatchetCudaError):
        e.step("a", [1, 2], [2])
    with pytest.raises(RatchetCudaError):
        e.step("a", [1] * 24)                          # beyond what a slot holds
    assert e.position("a") == 17                       # refused steps leave the sequence where it was
    e.end("a")
    e.end("a")
    assert e.position("b") == 0 and int(e.step("b", [3], [0])[0].argmax()) == 4


def test_requests_share_slots_first_come_first_served():
    e = Engine(CountingModel(), max_tokens=60, slots=2, portion=16)
    reqs = [Request([1, 2, 3], 9), Request([4], 1), Request(list(range(30)), 5), Request([7, 7], 12, stop=expected([7, 7], 3)[2])]
    done = e.run(reqs)
    assert [r.output for r in done[:3]] == [expected(r.prompt, r.max_new_tokens) for r in reqs[:3]]
    assert done[3].output == expected([7, 7], 3)
    assert e.generate([5, 6], 4) == expected([5, 6], 4)
    with pytest.raises(RatchetCudaError):
        e.run([Request([], 3)])
    with pytest.raises(RatchetCudaError):
        e.generate([1] * 59, 5)
    assert e.generate([9], 2) == expected([9], 2)      # a failed request gave its slot back


def test_sampler():
    z = np.array([0.0, 3.0, 2.9, -5.0], np.float32)
    assert Sampler().pick(z) == 1 and Sampler(temperature=1.0, top_k=1).pick(z) == 1
    s = Sampler(temperature=1.0, top_k=2, seed=1)
    picks = [s.pick(z) for _ in range(400)]
    assert set(picks) == {1, 2} and 0.4 < picks.count(1) / 400 < 0.65
    a, b = Sampler(0.7, 0, 5), Sampler(0.7, 0, 5)
    assert [a.pick(z) for _ in range(20)] == [b.pick(z) for _ in range(20)]
    with pytest.raises(RatchetCudaError):
        Sampler(temperature=-1.0)


# ---------------------------------------------------------------------------------------- the restatement itself
def test_restatement_state_carries_over():
    g = np.random.Generator(np.random.PCG64(1))
    q, k, v = g.standard_normal((9, 2, 3)), g.standard_normal((9, 2, 3)), g.standard_normal((9, 2, 4))
    o, s = dz.linear_attention(q, k, v, (0.4, 0.9))
    o1, s1 = dz.linear_attention(q[:4], k[:4], v[:4], (0.4, 0.9))
    o2, s2 = dz.linear_attention(q[4:], k[4:], v[4:], (0.4, 0.9), s1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(s, s2)
    direct = sum(0.9 ** (8 - j) * (k[j, 1] @ q[8, 1]) * v[j, 1] for j in range(9))
    assert np.allclose(o[8, 1], direct)


def test_restatement_is_causal_and_windowed():
    cfg = B.config(24, 20, [B.latent(2, 6, 4, 5, 8, 10, 4, 0.3, scaling=B.YARN, ff=9)])
    W = B.weights(cfg, 5)
    t = list(range(12))
    a = dz.forward(cfg, W, t)
    assert np.allclose(dz.forward(cfg, W, t[:7]), a[:7])
    changed = [t[0] + 7] + t[1:]
    b = dz.forward(cfg, W, changed)
    differs = np.abs(a - b).max(-1) > 1e-9
    assert differs[:4].all() and not differs[4:].any()
