"""Host side of the Mefesun decoder without a GPU: configuration, shared layers, visible rows; and the plain restatement's own
consistency."""
import json

import numpy as np
import pytest

from oracle import mefesun_plain as mp
from ratchet_b200 import RatchetCudaError, capi
from ratchet_b200.callers import GroupedMixer
from ratchet_b200.models import REGISTRY, MefesunConfig
from ratchet_b200.safetensors import SafetensorsFile

from . import mefesun_builders as B


def copy(cfg):
    return json.loads(json.dumps(cfg))


# ---------------------------------------------------------------------------------------- configuration
def test_configuration_is_read():
    assert "Mefesun" in REGISTRY
    for cfg in B.CONFIGS.values():
        c = MefesunConfig.read(copy(cfg))
        assert (c.width, c.vocab, c.eps, c.softcap) == (cfg["width"], cfg["vocab"], cfg["norm"]["eps"], cfg.get("logit_softcap"))
        assert list(c.weights_of) == [mp.owner(cfg, i) for i in range(len(cfg["layers"]))]
        for lc, e in zip(c.layers, cfg["layers"]):
            m = e["mixer"]
            assert (lc.mixer.heads, lc.mixer.kv_heads, lc.mixer.dim, lc.mixer.vdim, lc.mixer.chunk, lc.mixer.scale) == \
                (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["scale"])
            assert lc.mlp == bool(e["mlp"]) and lc.mixer.rot.dims == m["rot"]["dims"]
    assert MefesunConfig.read(copy(B.CONFIGS["mixed"])).weights_of == (0, 1, 0, 3, 0)
    free = copy(B.CONFIGS["odd"])
    del free["layers"][0]["mixer"]["mask"]
    assert MefesunConfig.read(free).layers[0].mixer.chunk == 0


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
                                    lambda c: c["layers"][3]["mlp"].update(kind="routed"), lambda c: c["layers"][2].update(weights_of=9),
                                    lambda c: c["layers"][2].update(weights_of=2), lambda c: c["layers"][2].update(weights_of=1),
                                    lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18),
                                    lambda c: c.update(logit_softcap=-1.0)])
def test_configurations_that_cannot_run_are_refused(change):
    cfg = copy(B.CONFIGS["mixed"])
    change(cfg)
    with pytest.raises(RatchetCudaError):
        MefesunConfig.read(cfg)


def test_model_folder_round_trip(tmp_path):
    cfg = B.CONFIGS["mixed"]
    W = B.weights(cfg, 2)
    f = SafetensorsFile(B.write_model(str(tmp_path), cfg, W) + "/model.safetensors")
    assert all(np.array_equal(f.f32(k), v) for k, v in W.items())
    assert not any(k.startswith(("l2.", "l4.")) for k in W)


def test_rows_seen_before_a_position():
    def mixer(window, chunk):
        return GroupedMixer(*[None] * 9, 1e-5, 1, 1, 2, 2, 1.0, window, chunk)
    for chunk in (1, 5, 64):
        assert [mixer(0, chunk).seen_before(p) for p in range(200)] == [sum(mp.same_chunk(p, j, chunk) for j in range(p)) for p in range(200)]
    assert [mixer(4, 0).seen_before(p) for p in range(6)] == [0, 1, 2, 3, 3, 3] and mixer(0, 0).seen_before(17) == 17


# ---------------------------------------------------------------------------------------- the restatement itself
def test_restatement_is_causal_and_chunked():
    cfg = B.config(24, 20, [B.attention(4, 2, 6, 5, 4, 0.3, dims=4, scaling=B.YARN, ff=9)])
    W = B.weights(cfg, 5)
    t = list(range(12))
    a = mp.forward(cfg, W, t)
    assert np.allclose(mp.forward(cfg, W, t[:7]), a[:7])
    for place, reach in ((0, 4), (3, 4), (4, 8), (6, 8)):
        changed = list(t)
        changed[place] += 7
        differs = np.abs(a - mp.forward(cfg, W, changed)).max(-1) > 1e-9
        assert not differs[:place].any() and differs[place:reach].all() and not differs[reach:].any()


def test_restatement_sink_and_groups():
    g = np.random.Generator(np.random.PCG64(4))
    q, k, v = g.standard_normal((6, 4, 3)), g.standard_normal((6, 2, 3)), g.standard_normal((6, 2, 5))
    sink = np.array([-50.0, 0.5, 2.0, 60.0])
    o = mp.sink_attention(q, k, v, 0.7, sink, None)
    p = np.exp(0.7 * k[:, 0] @ q[5, 1])                      # query heads 0 and 1 read key head 0
    assert np.allclose(o[5, 1], (p @ v[:, 0]) / (p.sum() + np.exp(0.5)))
    p = np.exp(0.7 * k[:, 0] @ q[5, 0])
    assert np.allclose(o[5, 0], (p @ v[:, 0]) / p.sum()) and np.abs(o[:, 3]).max() < 1e-20
    assert np.allclose(mp.softcap(np.array([-400.0, 0.1, 400.0]), 20.0), [-20.0, 0.1, 20.0], atol=1e-5)


@pytest.mark.parametrize("chunk", [3, 16])
def test_loud_models_show_who_sees_whom(chunk):
    """The weights the GPU tests use: a place that sees the loud token differs from one that does not by more than any tolerance."""
    cfg, W = B.loud_case(chunk)
    tokens = [2 + k % 30 for k in range(4 * chunk)]
    quiet = mp.forward(cfg, W, tokens)
    for at in (0, chunk - 1, chunk, 2 * chunk - 1):
        loud = mp.forward(cfg, W, tokens[:at] + [1] + tokens[at + 1:])
        shift = (loud - quiet).std(-1) / quiet.std(-1).mean()
        seen = np.array([mp.same_chunk(i, at, chunk) for i in range(len(tokens))])
        assert (shift[seen] > 0.2).all() and (shift[~seen] < 1e-12).all()


def test_linear_activation_names():
    assert capi.LINEAR_ACTS == {None: 0, "silu": 1, "relu_squared": 2, "softcap": 3}
