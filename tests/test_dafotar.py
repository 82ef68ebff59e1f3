"""Dafotar without a GPU: its configuration and description, what every run keeps per request (a run that reads another
run's keys keeps its convolution's inputs all the same; pages live as long as the widest window that reads them), and the
plain implementation's mechanisms against closed forms written here."""
import json
import math

import numpy as np
import pytest

import dafotar_util as du
from plain import dafotar_plain as plain


def spec_of(name):
    from air_b200.config import load_config
    from air_b200.parts import registry
    c = load_config(du.CONFIGS[name])
    return registry.architecture(c.architecture).build_spec(c)


def test_config_round_trip_and_description():
    from air_b200.config import load_config, ConfigError
    from air_b200.parts import registry
    from air_b200.engine.model import Model
    for name in ("A", "B", "C", "D", "E", "random2", "random5", "random9"):
        du.model_folder(name)
        cfg = du.CONFIGS[name]
        c = load_config(cfg)
        assert c.architecture == "Dafotar" and c.width == cfg["width"] and len(c.layers) == len(cfg["layers"])
        assert load_config(c.to_dict()) == c
        assert load_config(du.model_folder(name)) == c
        model = Model(registry.architecture(c.architecture).build_spec(c))
        names = {t.name: tuple(t.shape) for t in model.tensor_specs()}
        assert {n: a.shape for n, a in du.draw_tensors(cfg, 0).items()} == names

    def refused(change):
        bad = json.loads(json.dumps(du.CONFIGS["A"]))
        change(bad)
        with pytest.raises(ConfigError):
            load_config(bad)

    refused(lambda d: d["layers"][0].update(type="conv"))
    refused(lambda d: d.pop("norm"))
    refused(lambda d: d.pop("streams"))
    refused(lambda d: d.update(streams=0))
    refused(lambda d: d["layers"][1]["mixer"].pop("gate_cap"))
    refused(lambda d: d["layers"][0]["mixer"].update(kv_heads=4))            # six heads
    refused(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18))        # a head of 16
    refused(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    refused(lambda d: d["layers"][2]["mixer"].update(kv_from=1))             # an mlstm layer
    refused(lambda d: d["layers"][3]["mixer"].update(kv_from=2))             # a layer that borrows itself
    refused(lambda d: d["layers"][0]["mixer"].update(kv_from=2))             # a later layer
    refused(lambda d: d["layers"][2]["mixer"].update(vdim=24))               # other sizes than the layer it reads
    refused(lambda d: d["layers"][0]["mlp"].update(kind="moe"))


def test_what_every_run_keeps():
    from air_b200.engine.model import Model
    from air_b200.parts.base import PagedKV, SlotState
    spec = spec_of("A")
    assert [r.cache_from for r in spec.order] == [None, None, 0, 0, None]
    assert all(b.kind == "streams" for b in spec.layers) and spec.output_name is None
    first, wide, narrow = (spec.layers[i].parts["mixer"] for i in (0, 2, 3))
    assert (first["borrows"], wide["borrows"]) == (False, True)
    assert (first["window"], wide["window"], narrow["window"]) == (24, 50, 7)
    assert first["keep"] == wide["keep"] == narrow["keep"] == 50
    assert "feed_forward" not in spec.layers[2].parts and "feed_forward" in spec.layers[3].parts
    needs = Model(spec).cache_needs()
    conv = SlotState((3, 72))
    assert needs[0] == (PagedKV(2, 16, 50, 20), conv)
    assert needs[1] == (SlotState((3, 20, 12)), SlotState((3, 20)), SlotState((3,)), conv)
    assert needs[2] == needs[3] == (conv,)
    assert needs[5] == ()
    # one tap: nothing to keep; a layer that nobody borrows from keeps its own window
    spec = spec_of("B")
    needs = Model(spec).cache_needs()
    assert needs[1] == (PagedKV(1, 32, 1, 24),) and needs[2] == (PagedKV(4, 8, 1000, 16),) and needs[4] == ()
    spec = spec_of("E")
    assert spec.layers[3].parts["mixer"]["keep"] is None and spec.layers[2].parts["mixer"]["position"]["rotary_dim"] == 0
    assert spec.layers[2].parts["mixer"]["value_position"]["rotary_dim"] == 32


def test_pages_live_as_long_as_the_widest_window_that_reads_them():
    from air_b200.cache.manager import CacheManager
    from air_b200.engine.model import Model
    cache = CacheManager(Model(spec_of("A")).cache_needs(), 16, 12, 2, allocate=False)
    cache.open("a")
    for n in (40, 1, 60):
        cache.reserve([("a", n)])
        cache.commit("a", n)
    # 101 tokens: a query at 101 sees from 101 - 50 + 1 = 52 on, that is from block 3 of 7 on
    assert cache.used_pages("a") == 4
    cache.check()
    cache.close("a")
    assert cache.free_pages() == 12


def test_portions_and_chunks_of_the_matrix_memory():
    from air_b200.parts.base import HostBatch
    from air_b200.parts.recurrent import MLSTM
    from air_b200.parts.spec import PartSpec
    part = MLSTM(PartSpec("mlstm", dict(hidden=8, heads=1, head_dim=4, v_dim=4, gate_cap=3.0, eps=1e-6)))
    counts = [1, 130, 15, 16, 64]
    starts = np.concatenate([[0], np.cumsum(counts)]).tolist()
    plan = part.plan(HostBatch(counts=counts, lengths=[9, 0, 3, 70, 5], slots=[4, 2, 0, 3, 1], q_start=starts))
    assert plan.values == {"long": True, "short": True}
    assert plan.arrays["short_slots"].tolist() == [4, -1, 0, -1, -1]
    assert plan.arrays["portions"].tolist() == [[1, 130, 2, 0], [146, 16, 3, 3], [162, 64, 1, 4]]
    assert plan.arrays["chunks"].tolist() == [[1, 64], [65, 64], [129, 2], [146, 16], [162, 64]]
    plan = part.plan(HostBatch(counts=[1, 2], lengths=[0, 0], slots=[0, 1], q_start=[0, 1, 3]))
    assert plan.values == {"long": False, "short": True} and plan.arrays["chunks"].shape == (0, 2)


def test_plain_mechanisms_against_closed_forms():
    rng = np.random.default_rng(0)
    # layer norm: shifting and scaling a row changes nothing but through eps; the bias is added behind
    x = rng.normal(size=(3, 8))
    y = plain.layer_norm(x, np.ones(8), np.zeros(8), 0.0)
    assert np.allclose(y.mean(-1), 0) and np.allclose((y * y).mean(-1), 1)
    assert np.allclose(plain.layer_norm(5 * x + 7, 2 * np.ones(8), np.full(8, 3.0), 0.0), 2 * y + 3)
    # streams: mix is indexed from, to
    X = rng.normal(size=(2, 4, 3))
    out = plain.mix_streams(X, np.array([[0.0, 1.0], [0.0, 0.0]]), np.array([0.0, 2.0]), np.ones((4, 3)))
    assert np.allclose(out[0], 0) and np.allclose(out[1], X[0] + 2)
    assert np.allclose(plain.read_streams(X, np.array([2.0, -1.0])), 2 * X[0] - X[1])
    # the convolution: the input itself, the last tap on the token, zeros ahead of the sequence
    h = rng.normal(size=(5, 2))
    w = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 0.0]])
    y = plain.input_convolution(h, w)
    assert np.allclose(y[0, 0], 101 * h[0, 0]) and np.allclose(y[1, 0], 10 * h[0, 0] + 101 * h[1, 0])
    assert np.allclose(y[4, 0], h[2, 0] + 10 * h[3, 0] + 101 * h[4, 0]) and np.allclose(y[:, 1], h[:, 1])
    # rotation: first and second half pair up; the rest passes; turning forth and back is nothing
    v = rng.normal(size=(4, 2, 6))
    t = plain.turn(v, [0, 1, 5, 9], 4, 10.0, np.float64)
    assert np.allclose(t[0], v[0]) and np.allclose(t[..., 4:], v[..., 4:])
    f = 10.0 ** -0.5
    assert np.allclose(t[2, 1, 1], v[2, 1, 1] * math.cos(5 * f) - v[2, 1, 3] * math.sin(5 * f))
    assert np.allclose(t[2, 1, 3], v[2, 1, 3] * math.cos(5 * f) + v[2, 1, 1] * math.sin(5 * f))
    assert np.allclose(plain.turn(t, [0, 1, 5, 9], 4, 10.0, np.float64, sign=-1.0), v)
    # a window of two: the token and the one before it
    q, k = np.zeros((4, 1, 2)), np.zeros((4, 1, 2))
    v = np.arange(4.0).reshape(4, 1, 1)
    assert np.allclose(plain.window_attention(q, k, v, [1.0], 2)[:, 0, 0], [0.0, 0.5, 1.5, 2.5])
    assert np.allclose(plain.window_attention(q, k, v, [1.0], 1)[:, 0, 0], [0.0, 1.0, 2.0, 3.0])
    assert np.allclose(plain.window_attention(q, k, v, [1.0], None)[3, 0, 0], 1.5)
    # the matrix memory with its weights written out: no running maximum, everything relative to exp(0)
    T, d, dv = 6, 3, 2
    q, k, v = rng.normal(size=(T, 1, d)), rng.normal(size=(T, 1, d)), rng.normal(size=(T, 1, dv))
    i, f = rng.normal(size=(T, 1)) * 2, -rng.uniform(0.1, 2.0, size=(T, 1))
    o = plain.mlstm_memory(q, k, v, i, f, np.float64)
    C = n = 0.0
    m = 0.0
    for s in range(T):
        weight = math.exp(i[s, 0] + f[s + 1:, 0].sum())
        C, n = C + weight * np.outer(k[s, 0], v[s, 0]), n + weight * k[s, 0]
        m = max(m + f[s, 0], i[s, 0])
    want = (C.T @ q[-1, 0]) * math.exp(-m) / (max(abs(n @ q[-1, 0]) * math.exp(-m), math.exp(-m)) + 1e-6)
    assert np.allclose(o[-1, 0], want)
    # the floor: with one faint token the denominator is exp(-m), m having started at zero
    o = plain.mlstm_memory(np.ones((1, 1, 1)), np.full((1, 1, 1), 1e-3), np.ones((1, 1, 1)), np.full((1, 1), -1.0),
                           np.full((1, 1), -0.5), np.float64)
    assert np.allclose(o, 1e-3 * math.exp(-0.5) / (math.exp(0.5) + 1e-6))
    assert np.allclose(plain.dense_ff({"f.gate": np.array([[1.0, -1.0]]), "f.up": np.array([[0.0, 1.0]]),
                                       "f.down": np.array([[3.0], [4.0]])}, "f.", np.array([[5.0, 2.0], [1.0, 2.0]])),
                       [[18.0, 24.0], [0.0, 0.0]])


def test_oracle_in_32_bit_is_close_to_itself_in_64():
    for name in ("A", "E"):
        cfg, tensors = du.plain_model(name)
        toks = du.tokens_for(name, 60, 1)
        a = plain.forward(cfg, tensors, toks)
        b = plain.forward(cfg, tensors, toks, dtype=np.float32)
        assert np.abs(a - b).max() < 2e-5 * np.abs(a).max()


def test_every_mechanism_of_the_test_models_matters():
    """Leaving one mechanism out of the oracle moves the logits far beyond what rounding does: a test that passes
    would not pass with the mechanism missing."""
    cfg, tensors = du.plain_model("A")
    toks = du.tokens_for("A", 90, 3)
    ref = plain.forward(cfg, tensors, toks)
    scale = np.abs(ref).max()

    def moved(change):
        c, t = json.loads(json.dumps(cfg)), dict(tensors)
        change(c, t)
        return np.abs(plain.forward(c, t, toks) - ref).max() / scale

    ones = lambda t, n: t.update({n: np.ones_like(t[n])})
    zeros = lambda t, n: t.update({n: np.zeros_like(t[n])})
    for n in (25, 23):
        assert moved(lambda c, t: c["layers"][0]["mixer"]["mask"].update(size=n)) > 0.005
    for n in (49, 51):
        assert moved(lambda c, t: c["layers"][2]["mixer"]["mask"].update(size=n)) > 0.005
    assert moved(lambda c, t: c["layers"][0]["mixer"]["rot"].update(base=5000.0)) > 0.005
    assert moved(lambda c, t: c["layers"][0]["mixer"]["rot"].update(dims=16)) > 0.005
    assert moved(lambda c, t: ones(t, "l0.mix.temp")) > 0.005
    assert moved(lambda c, t: ones(t, "l2.mix.q.norm")) > 0.005
    assert moved(lambda c, t: zeros(t, "l1.canon1")) > 0.005
    assert moved(lambda c, t: t.update({"l1.canon1": np.roll(t["l1.canon1"], 1, axis=1)})) > 0.005
    assert moved(lambda c, t: zeros(t, "l0.norm2.b")) > 0.005
    assert moved(lambda c, t: t.update({"l1.hc1.mix": t["l1.hc1.mix"].T})) > 0.005
    assert moved(lambda c, t: t.update({"l1.hc2.in": t["l1.hc2.in"][::-1]})) > 0.005
    assert moved(lambda c, t: t.update({"l1.hc1.out": t["l1.hc1.out"][::-1]})) > 0.005
    assert moved(lambda c, t: c["layers"][1]["mixer"].update(gate_cap=50.0)) > 0.005
    assert moved(lambda c, t: zeros(t, "l1.mix.i.b")) > 0.005
    assert moved(lambda c, t: zeros(t, "l4.mix.f.b")) > 0.005
    assert moved(lambda c, t: zeros(t, "l4.mix.i")) > 0.005
