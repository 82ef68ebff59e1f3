"""Sesulorn without a GPU: its configuration and description, what every run keeps per request, the distance table's rows,
and the plain implementation's mechanisms against closed forms written here."""
import json
import math

import numpy as np
import pytest

import sesulorn_util as su
from plain import sesulorn_plain as plain


def spec_of(name):
    from air_b200.config import load_config
    from air_b200.parts import registry
    c = load_config(su.CONFIGS[name])
    return registry.architecture(c.architecture).build_spec(c)


def test_config_round_trip_and_description():
    from air_b200.config import load_config, ConfigError
    from air_b200.parts import registry
    from air_b200.engine.model import Model
    for name in ("A", "B", "C", "D", "E", "random2", "random5", "random9", "random12"):
        su.model_folder(name)
        cfg = su.CONFIGS[name]
        c = load_config(cfg)
        assert c.architecture == "Sesulorn" and c.width == cfg["width"] and len(c.layers) == len(cfg["layers"])
        assert load_config(c.to_dict()) == c
        assert load_config(su.model_folder(name)) == c, "the sizes that only the tensors' shapes give"
        model = Model(registry.architecture(c.architecture).build_spec(c))
        names = {t.name: tuple(t.shape) for t in model.tensor_specs()}
        assert {n: a.shape for n, a in su.draw_tensors(cfg, 0).items()} == names

    def refused(change):
        bad = json.loads(json.dumps(su.CONFIGS["A"]))
        change(bad)
        with pytest.raises(ConfigError):
            load_config(bad)

    refused(lambda d: d["layers"][0].update(type="conv"))
    refused(lambda d: d.pop("norm"))
    refused(lambda d: d["loop"].update(stop=9))
    refused(lambda d: d["loop"].update(times=0))
    refused(lambda d: d["layers"][0]["mixer"].update(kv_heads=4))            # six heads
    refused(lambda d: d["layers"][0]["mixer"].update(bias_max=4))            # half of the table's rows
    refused(lambda d: d["layers"][0]["mixer"].pop("buckets"))
    refused(lambda d: d["layers"][1]["mixer"].pop("decay_rank"))
    refused(lambda d: d["layers"][1]["mixer"].update(conv=0))
    refused(lambda d: d["layers"][2]["mixer"]["rot"].update(dims=4))         # a rotated part of 8
    refused(lambda d: d["layers"][2]["mixer"].update(q_rank=0))
    refused(lambda d: d["layers"][0]["mlp"]["router"].update(top=5))         # two groups of two
    refused(lambda d: d["layers"][0]["mlp"]["expert"].pop("limit"))
    refused(lambda d: d["layers"][0]["mlp"].update(kind="wide"))


def test_what_every_run_keeps_and_where_passes_begin():
    from air_b200.engine.model import Model
    from air_b200.parts.base import PagedKV, PagedLatent, SlotState
    spec = spec_of("A")
    assert [r.layer for r in spec.order] == [0, 1, 0, 1, 0, 1, 2, 3, 4]
    assert [r.mix_embedding for r in spec.order] == ["loop.in", None] * 3 + [None] * 3
    assert all(r.cache_from is None for r in spec.order) and spec.stream_mixes == ("loop.in",)
    model = Model(spec)
    assert model.embedding_copies == 2
    needs = model.cache_needs()
    state = (SlotState((4, 20, 12)), SlotState((2 * 2 * 20 + 4 * 12, 3)))
    for run in (0, 2, 4):
        assert needs[run] == (PagedKV(2, 16, None, 20),) and needs[run + 1] == state
    assert needs[6] == (PagedLatent(48),) and needs[8] == (PagedKV(3, 24, None, 8),) and needs[9] == ()
    spec = spec_of("B")
    assert spec.stream_mixes == () and Model(spec).embedding_copies == 1
    assert [r.layer for r in spec.order] == [0, 1, 2, 3, 4]
    assert [r.layer for r in spec_of("C").order] == [0, 1, 2, 1, 2]
    # a stretch of no layers: its matrix is in the model file, nothing runs through it
    from air_b200.config import load_config
    from air_b200.parts import registry
    c = load_config(dict(su.CONFIGS["A"], loop=dict(start=2, stop=2, times=3)))
    spec = registry.architecture(c.architecture).build_spec(c)
    assert [r.layer for r in spec.order] == [0, 1, 2, 3, 4] and not any(r.mix_embedding for r in spec.order)
    assert "loop.in" in {t.name for t in Model(spec).tensor_specs()}


@pytest.mark.parametrize("rows,span", [(8, 40), (2, 3), (2, 2), (32, 128), (32, 256), (16, 300), (10, 6), (6, 30.5), (14, 60),
                                       (64, 1000), (9, 17)])
def test_rows_of_the_distance_table(rows, span):
    """The spread-out rows against the plain function, far past the table's reach; every edge between two rows is where
    the logarithm says (checked with the inequality's two sides, not with the logarithm)."""
    from air_b200.parts.normed_attention import distance_rows
    spread = distance_rows(rows, span)
    for n in range(0, 4 * int(span) + 10):
        assert spread[min(n, len(spread) - 1)] == plain.bucket(n, rows, span), n
    assert spread[-1] == rows - 1 and (len(spread) == 1 or spread[-2] < rows - 1)
    low = rows // 2
    for n in range(low, len(spread)):
        k = spread[n] - low
        lo, hi = low * (span / low) ** (k / (rows - low)), low * (span / low) ** ((k + 1) / (rows - low))
        assert n >= lo * (1 - 1e-12) and (spread[n] == rows - 1 or n < hi * (1 + 1e-12)), (n, k)
    assert spread[:low] == list(range(low))


def test_plain_mechanisms_against_closed_forms():
    rng = np.random.default_rng(0)
    # layer norm: no mean, unit variance, then weight and bias
    x = rng.normal(size=(3, 8))
    y = plain.layer_norm(x, np.ones(8), np.zeros(8), 0.0)
    assert np.allclose(y.mean(axis=1), 0) and np.allclose((y * y).mean(axis=1), 1)
    assert np.allclose(plain.layer_norm(5 * x + 7, 2 * np.ones(8), np.full(8, 3.0), 0.0), 2 * y + 3)
    # the distance table: eight rows over 32 positions; behind 4 the row grows by one with every factor 8^(1/4)
    assert [plain.bucket(n, 8, 32) for n in (0, 3, 4, 6, 7, 11, 12, 19, 20, 31, 32, 1000)] == \
        [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    # attention with nothing but the bias: softmax of the table's numbers; the scale does not touch them
    T = 6
    zero, v = np.zeros((T, 2, 4)), np.arange(6.0).reshape(T, 1, 1)
    table = np.array([[0.0, 1.0], [2.0, 0.0], [-1.0, 5.0], [0.5, 0.0]])
    o = plain.biased_attention(zero, np.zeros((T, 1, 4)), v, 7.0, table, 4)
    rows = [plain.bucket(n, 4, 4) for n in range(T)]
    for h in range(2):
        e = np.exp([table[rows[5 - j], h] for j in range(T)])
        assert np.allclose(o[5, h, 0], (e * np.arange(6.0)).sum() / e.sum()) and np.allclose(o[0, h, 0], 0.0)
    # the convolution: the last tap on the token, zeros ahead of the sequence
    h = rng.normal(size=(5, 2))
    w = np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 0.0]])
    y = plain.short_convolution(h, w)
    assert np.allclose(y[0, 0], 100 * h[0, 0]) and np.allclose(y[1, 0], 10 * h[0, 0] + 100 * h[1, 0])
    assert np.allclose(y[4, 0], h[2, 0] + 10 * h[3, 0] + 100 * h[4, 0]) and np.allclose(y[:, 1], 0)
    # the delta rule: without decay, with b = 1 and one unit key written twice, the read-out is the last value
    one = np.ones((2, 1, 3))
    k = np.zeros((2, 1, 3))
    k[:, 0, 1] = 1.0
    v = rng.normal(size=(2, 1, 4))
    assert np.allclose(plain.delta_memory(k, k, v, one, np.ones((2, 1)), np.float64)[:, 0], v[:, 0])
    # ... and the decay works on the key's channel before the value is compared: S = g k v0^T, u = v1 - g v0
    g = np.full((2, 1, 3), 0.25)
    assert np.allclose(plain.delta_memory(k, k, v, g, np.full((2, 1), 0.5), np.float64)[1, 0],
                       0.25 * 0.5 * v[0, 0] + 0.5 * (v[1, 0] - 0.25 * 0.5 * v[0, 0]))
    other = np.ones((2, 1, 3))
    other[:, 0, 1] = 0.0                     # the channel that the key lives in forgets everything
    assert np.allclose(plain.delta_memory(k, k, v, other, np.full((2, 1), 0.5), np.float64)[1, 0], 0.5 * v[1, 0])
    # decays: softplus(0) = ln 2, so g = 2^(-exp(A))
    w = {"a1": np.zeros((2, 5)), "a2": np.zeros((6, 2)), "dt_bias": np.zeros(6), "A_log": np.log([1.0, 3.0])}
    assert np.allclose(plain.channel_decay(w, "", np.ones((1, 5)), 2, 3), [[[0.5] * 3, [0.125] * 3]])
    # rotation: neighbours pair up
    v = rng.normal(size=(4, 2, 4))
    t = plain.turn_neighbours(v, 10.0, np.float64)
    f = 10.0 ** -0.5
    assert np.allclose(t[0], v[0]) and np.allclose(t[3, 1, 2], v[3, 1, 2] * math.cos(3 * f) - v[3, 1, 3] * math.sin(3 * f))
    assert np.allclose(t[3, 1, 3], v[3, 1, 3] * math.cos(3 * f) + v[3, 1, 2] * math.sin(3 * f))
    assert np.allclose(t[2, 0, 0], v[2, 0, 0] * math.cos(2) - v[2, 0, 1] * math.sin(2))
    # the router: the best expert marks a group (0.3 + 0.3 would mark the first one higher)
    s = np.array([0.3, 0.3, 0.35, 0.01, 0.02, 0.02])
    assert plain.chosen_experts(s, 3, 1, 2) == [2, 3] and plain.chosen_experts(s, 3, 2, 3) == [2, 0, 1]
    assert plain.chosen_experts(s, 1, 1, 2) == [2, 0]
    # experts: limits on both sides of the linear branch, one on the gate's
    w = {"e.gate": np.array([[1.0]]), "e.up": np.array([[2.0]]), "e.down": np.array([[3.0]])}
    act = lambda a: a / (1 + math.exp(-1.702 * a))
    for z, a, b in ((0.3, 0.3, 0.6), (5.0, 1.0, 1.0), (-4.0, -4.0, -1.0)):
        assert np.allclose(plain.clamped_expert(w, "e.", np.array([[z]]), 1.0), 3 * act(a) * (b + 1))
    assert plain.layer_order(dict(layers=[0] * 3, loop=dict(start=1, stop=2, times=2))) == \
        [(0, False), (1, True), (1, True), (2, False)]


def test_oracle_in_32_bit_is_close_to_itself_in_64():
    for name in ("A", "E"):
        cfg, tensors = su.plain_model(name)
        toks = su.tokens_for(name, 60, 1)
        a = plain.forward(cfg, tensors, toks)
        b = plain.forward(cfg, tensors, toks, dtype=np.float32)
        assert np.abs(a - b).max() < 2e-5 * np.abs(a).max()


def test_every_mechanism_of_the_test_models_matters():
    """Leaving one mechanism out of the oracle moves the logits far beyond what rounding does: a test that passes
    would not pass with the mechanism missing."""
    cfg, tensors = su.plain_model("A")
    toks = su.tokens_for("A", 90, 3)
    ref = plain.forward(cfg, tensors, toks)
    scale = np.abs(ref).max()

    def moved(change):
        c, t = json.loads(json.dumps(cfg)), dict(tensors)
        change(c, t)
        return np.abs(plain.forward(c, t, toks) - ref).max() / scale

    ones = lambda t, n: t.update({n: np.ones_like(t[n])})
    zeros = lambda t, n: t.update({n: np.zeros_like(t[n])})
    mixer = lambda c, i: c["layers"][i]["mixer"]
    for n in ("l0.mix.rel", "l0.mix.q.b", "l0.mix.v.b", "l0.norm1.b", "l1.mix.a2", "l1.mix.g2", "l1.mix.b", "l1.mix.A_log",
              "l1.mix.dt_bias", "l2.mix.dq", "l0.mlp.shared.sg", "final.norm.b", "l4.mix.rel"):
        assert moved(lambda c, t: zeros(t, n)) > 0.005, n
    for n in ("l1.mix.norm", "l2.mix.dq.norm", "l2.mix.dkv.norm", "l1.norm1"):
        assert moved(lambda c, t: ones(t, n)) > 0.005, n
    assert moved(lambda c, t: mixer(c, 0).update(bias_max=30)) > 0.005
    assert moved(lambda c, t: t.update({"l0.mix.rel": np.roll(t["l0.mix.rel"], 1, axis=0)})) > 0.005
    assert moved(lambda c, t: mixer(c, 0).update(scale=0.45)) > 0.005
    assert moved(lambda c, t: mixer(c, 2)["rot"].update(base=5000.0)) > 0.005
    assert moved(lambda c, t: t.update({"l1.mix.q.conv": np.roll(t["l1.mix.q.conv"], 1, axis=1)})) > 0.005
    assert moved(lambda c, t: c["loop"].update(times=2)) > 0.005
    assert moved(lambda c, t: t.update({"loop.in": t["loop.in"] * np.repeat([1.0, 0.0], cfg["width"])})) > 0.005
    assert moved(lambda c, t: c["layers"][0]["mlp"]["expert"].update(limit=2.0)) > 0.005
    assert moved(lambda c, t: c["layers"][0]["mlp"]["shared"].update(limit=1.2)) > 0.005
    assert moved(lambda c, t: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3)) > 0.005
    assert moved(lambda c, t: c["layers"][3]["mlp"]["router"].update(top=2)) > 0.005
    assert moved(lambda c, t: c["norm"].update(eps=1e-2)) > 0.0005
