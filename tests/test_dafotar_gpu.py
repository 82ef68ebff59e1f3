"""Dafotar on the GPU against the plain implementation (tests/plain/dafotar_plain.py, 64-bit): every mechanism alone
through its part or kernel, then whole models through Engine.step, the scheduler and the trace runner, in float32 and
bfloat16, for configurations that differ in every size and option (dafotar_util.CONFIGS)."""
import tempfile
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import dafotar_util as du
import util
from plain import dafotar_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.ascontiguousarray(a)).to(device=DEV, dtype=dtype)


def i32(a):
    return torch.tensor(list(a), dtype=torch.int32, device=DEV)


def runtime(dtype, page=16):
    from air_b200.parts.base import Runtime
    return Runtime(torch.device(DEV), DT[dtype], page, status=torch.zeros(1, dtype=torch.int32, device=DEV))


def context_for(cache, entries, *parts):
    from air_b200.engine.batch import Entry, build_context
    entries = [Entry(*e) for e in entries]
    for e in entries:
        if e.request not in cache.sequences:
            cache.open(e.request)
    cache.reserve([(e.request, len(e.tokens)) for e in entries])
    planners = {p.plan_key(): p for p in parts if p.plan_key() is not None}
    return build_context(entries, cache, DEV, status=torch.zeros(1, dtype=torch.int32, device=DEV),
                         planners=list(planners.values()))


def summed(y):
    return (y.sum(0) if y.dim() == 3 else y).float().cpu().numpy()


def rounded(w, dtype):
    return {k: du.bf16(a).astype(np.float64) for k, a in w.items()} if dtype == "bfloat16" else w


WIDE = ("q.norm", "k.norm", "temp", "i.b", "f.b", "norm")


def load(part, w, dtype, page=16, prefix="m."):
    part.load({prefix + k: dev(a, torch.float32 if k in WIDE else DT[dtype]) for k, a in w.items()}, runtime(dtype, page))
    return part


def run_in_steps(run, cache, streams, steps):
    """streams: request -> inputs [T, E]; steps: lists of (request, tokens); run(x, entries) -> outputs.  Returns
    request -> outputs [T, E]."""
    done = {r: 0 for r in streams}
    outs = {r: [] for r in streams}
    for step in steps:
        x = np.concatenate([streams[r][done[r]:done[r] + n] for r, n in step])
        y = run(x, [(r, [0] * n, []) for r, n in step])
        at = 0
        for r, n in step:
            outs[r].append(y[at:at + n])
            cache.commit(r, n)
            done[r] += n
            at += n
    assert all(done[r] == len(streams[r]) for r in streams)
    return {r: np.concatenate(o) for r, o in outs.items()}


STEPS = [[("a", 3)], [("a", 61), ("b", 1)], [("b", 2), ("a", 1)], [("a", 150), ("b", 40)], [("a", 2)], [("a", 1), ("b", 1)],
         [("b", 30), ("a", 1)], [("a", 30)], [("a", 70), ("b", 1)], [("a", 1)]]          # a: 320 tokens, b: 75


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("S,T,E,parts", [(1, 13, 72, 1), (2, 5, 90, 3), (3, 300, 256, 2), (4, 2, 2048, 4), (5, 7, 64, 1),
                                         (16, 9, 48, 2), (3, 6, 10, 1), (2, 700, 4160, 1)])
def test_streams_completed_read_and_normalised(S, T, E, parts, dtype):
    """x'_t = sum_s mix x_s + out_t y, u = sum read x', layer norm of u: with the streams still one tensor and apart, the
    output as a tensor and as partial sums, for chosen rows (the streams stay), and completed alone."""
    from air_b200.parts.base import Norm, StreamSum
    from air_b200.parts.norm import LayerNorm
    from air_b200.parts.spec import PartSpec
    rng = np.random.default_rng(S * T + E)
    eps = 1e-5
    part = LayerNorm(PartSpec("layer", {"size": E, "eps": eps, "tensor": "", "bias": ".b"}), "n")
    w, b = rng.normal(1.0, 0.3, size=E), rng.normal(0.0, 0.5, size=E)
    part.load({"n": dev(w), "n.b": dev(b)}, runtime(dtype))
    tol = 2e-5 if dtype == "float32" else 2e-2
    close = lambda a, want, t: np.abs(a.float().cpu().numpy() - want).max() < t * np.abs(want).max()
    for equal in (True, False):
        X = rng.normal(size=(S, T, E)) * 3 + rng.normal(size=(S, T, 1)) * 5          # rows with a mean far from zero
        X = np.repeat(X[:1], S, axis=0) if equal else X
        y, mix = rng.normal(size=(parts, T, E)) * 2, rng.normal(size=(S, S)) / S
        out_w, read = rng.normal(size=S), rng.uniform(0.5, 1.5, size=S)
        hd = lambda: dev(X[0] if equal else X)
        delta = StreamSum(dev(y if parts > 1 else y[0]), dev(mix), dev(out_w))
        after = plain.mix_streams(X, mix, out_w, y.sum(0))
        h, rows = part.forward_streams(hd(), delta, dev(read))
        assert tuple(h.shape) == (S, T, E) and close(h, after, 2e-5)
        assert close(rows, plain.layer_norm(plain.read_streams(after, read), w, b, eps), tol)
        h0 = hd()
        same, rows = part.forward_streams(h0, None, dev(read))
        assert same is h0 and close(rows, plain.layer_norm(plain.read_streams(X, read), w, b, eps), tol)
        last = plain.layer_norm(after.sum(0), w, b, eps)
        pick = [T - 1, 0, T // 2]
        h0 = hd()
        assert close(part.forward(h0, delta, rows=i32(pick)), last[pick], tol)
        assert np.array_equal(h0.cpu().numpy(), hd().cpu().numpy())
        assert close(Norm.add_delta(hd(), delta), after, 2e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_norm_of_an_ordinary_stream(dtype):
    """The same norm for designs with one residual stream: every form in which an output can be handed on."""
    from air_b200.parts.base import GatedSum, NormedSum, ScaledSum
    from air_b200.parts.norm import LayerNorm
    from air_b200.parts.spec import PartSpec
    rng = np.random.default_rng(3)
    T, E, eps = 11, 136, 1e-6
    part = LayerNorm(PartSpec("layer", {"size": E, "eps": eps}), "n.")
    w, b = rng.normal(1.0, 0.3, size=E), rng.normal(0.0, 0.5, size=E)
    part.load({"n.weight": dev(w), "n.bias": dev(b)}, runtime(dtype))
    h, y, s = rng.normal(size=(T, E)) + 4, rng.normal(size=(3, T, E)), rng.normal(size=E)
    gate = rng.uniform(size=T)
    tol = 2e-5 if dtype == "float32" else 2e-2
    for delta, want in ((None, h), (dev(y[0]), h + y[0]), (dev(y), h + y.sum(0)), (dev(y[0], torch.bfloat16), h + du.bf16(y[0])),
                        (ScaledSum([(dev(y[0]), dev(s)), (dev(y[1]), None)]), h + s * y[0] + y[1]),
                        (GatedSum(dev(y[0]), dev(y[1]), dev(gate)), h + y[0] + gate[:, None] * y[1]),
                        (NormedSum(dev(y[0]), dev(s), 1e-5), h + plain.over_rms(y[0], 1e-5) * s)):
        for rows in (None, [3, 0, 10]):
            hd = dev(h)
            got = part.forward(hd, delta, rows=None if rows is None else i32(rows)).float().cpu().numpy()
            ref = plain.layer_norm(want, w, b, eps)
            assert np.abs(got - (ref if rows is None else ref[rows])).max() < tol * np.abs(ref).max()
            assert np.abs(hd.cpu().numpy() - (want if rows is None else h)).max() < 2e-5 * np.abs(want).max()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,taps", [(72, 4), (64, 1), (90, 6), (256, 3), (30, 2), (48, 19)])
def test_convolution_added_to_its_input_through_portions_slots_and_single_tokens(E, taps, dtype):
    """Two requests in steps that hold both; portions shorter than the taps; single tokens through the norm's own kernel
    (a step in which every row is its request's only token); a slot that another request held starts from zeros."""
    from air_b200.cache.manager import CacheManager
    from air_b200.parts.norm import LayerNorm
    from air_b200.parts.row_filter import ResidualConvolution
    from air_b200.parts.spec import PartSpec
    rng = np.random.default_rng(E + taps)
    eps = 1e-6
    w, b = rng.normal(1.0, 0.3, size=E), rng.normal(0.0, 0.5, size=E)
    norm = LayerNorm(PartSpec("layer", {"size": E, "eps": eps, "tensor": "", "bias": ".b"}), "n")
    norm.load({"n": dev(w), "n.b": dev(b)}, runtime(dtype))
    cw = rng.normal(size=(E, taps)) / taps ** 0.5
    conv = ResidualConvolution(PartSpec("residual_conv", {"size": E, "taps": taps}), "c")
    conv.load({"c": dev(cw)}, runtime(dtype))
    cache = CacheManager([conv.cache_needs()], 16, 40, 3, device=DEV)
    cache.open("other")
    single = []

    def run(x, entries):
        ctx = context_for(cache, entries)
        fused = conv.single_tokens(ctx, cache.views(0))
        single.append(fused is not None)
        _, y = norm.forward_streams(dev(x), None, dev(np.ones(1)), conv=fused, dtype=None if fused else torch.float32)
        return summed(y if fused else conv.forward(y, ctx, cache.views(0)))

    streams = {"a": rng.normal(size=(320, E)), "b": rng.normal(size=(75, E))}
    want = {r: plain.input_convolution(plain.layer_norm(x, w, b, eps), cw) for r, x in streams.items()}
    tol = 2e-5 if dtype == "float32" else 2e-2
    got = run_in_steps(run, cache, streams, STEPS)
    assert any(single) and not all(single)
    for r in streams:
        assert np.abs(got[r] - want[r]).max() < tol * np.abs(want[r]).max()
    cache.close("b")
    again = run_in_steps(run, cache, {"c": streams["b"]}, [[("c", 1)], [("c", 5)], [("c", 69)]])       # b's slot
    assert np.abs(again["c"] - want["b"]).max() < tol * np.abs(want["b"]).max()


def attention_weights(rng, E, m, dtype):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    sharp = (2.5 / (m["scale"] * d ** 0.5)) ** 0.5
    w = {"q": rng.normal(size=(H * d, E)) / E ** 0.5, "k": rng.normal(size=(G * d, E)) / E ** 0.5,
         "v": rng.normal(size=(G * dv, E)) / E ** 0.5, "o": rng.normal(size=(E, H * dv)) / (H * dv) ** 0.5,
         "q.norm": sharp * rng.normal(1.0, 0.15, size=d), "k.norm": sharp * rng.normal(1.0, 0.15, size=d),
         "temp": rng.uniform(0.6, 1.5, size=H)}
    return rounded(w, dtype)


def attention_part(E, m, eps, keep=None, borrows=False, prefix="m."):
    from air_b200.parts.normed_attention import NormedAttention
    from air_b200.parts.spec import PartSpec
    r = m.get("rot") or {}
    turned = lambda n: PartSpec("rope_live", {"rotary_dim": n if r else 0, "theta": r.get("base", 1.0), "pairing": "half"})
    window = m["mask"]["size"] if m.get("mask") else None
    return NormedAttention(PartSpec("normed_attention", {
        "hidden": E, "heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"],
        "scale": m["scale"], "window": window, "eps": eps, "qk_norm": "head", "head_temp": True,
        "position": turned(r.get("dims", 0)), "value_position": turned(m["vdim"]), "borrows": borrows,
        "keep": keep or window}), prefix)


ATTENTION = [      # heads, kv_heads, dim, vdim, scale, window, rotated dims, base, window of the layer that borrows, page
    (6, 2, 16, 20, 0.3, 24, 8, 500.0, 50, 16),
    (4, 4, 8, 16, 0.4, 33, 4, 100.0, 7, 16),
    (1, 1, 32, 24, 0.2, 1, 32, 10000.0, 2, 32),
    (3, 1, 14, 10, 0.3, 17, 6, 1000.0, 16, 16),
    (4, 2, 64, 64, 0.125, 64, 32, 10000.0, 65, 64),
    (4, 1, 128, 128, 0.09, 100, 128, 1000000.0, 63, 32),
    (2, 2, 32, 40, 0.2, None, 0, 10000.0, 200, 16),
    (8, 2, 64, 64, 0.2, 300, 0, 0, None, 16),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,scale,window,dims,base,other,page", ATTENTION)
def test_attention_and_a_layer_that_reads_its_keys(H, G, d, dv, scale, window, dims, base, other, page, dtype):
    """A layer and one behind it that reads its keys and values with queries, window and factors of its own, over two
    requests in steps that hold both, against the plain function on each whole sequence; pages that no window needs have
    gone back to the pool meanwhile, and slots and pages are used again."""
    from air_b200.cache.manager import CacheManager
    E, eps = 80, 1e-5
    rng = np.random.default_rng(H * d + dv)
    m = du.attention(H, G, d, dv, scale, window, dims, base)["mixer"]
    m2 = du.attention(H, G, d, dv, scale * 1.2, other, dims, base)["mixer"]
    w, w2 = attention_weights(rng, E, m, dtype), attention_weights(rng, E, m2, dtype)
    w2 = {k: a for k, a in w2.items() if k not in ("k", "v", "k.norm")}
    streams = {"a": rng.normal(size=(320, E)), "b": rng.normal(size=(75, E))}
    if dtype == "bfloat16":
        streams = {r: du.bf16(x).astype(np.float64) for r, x in streams.items()}
    wp = {"m." + k: a for k, a in w.items()}
    wp2 = {"n." + k: a for k, a in w2.items()}
    want = {}
    for r, x in streams.items():
        y, kv = plain.mixer_attention(wp, "m.", x, m, np.arange(len(x)), eps, np.float64)
        y2, _ = plain.mixer_attention(wp2, "n.", x, m2, np.arange(len(x)), eps, np.float64, shared=kv)
        want[r] = np.concatenate([y, y2], axis=1)
    keep = None if None in (window, other) else max(window, other)
    own = load(attention_part(E, m, eps, keep), w, dtype, page)
    reader = load(attention_part(E, m2, eps, keep, borrows=True, prefix="n."), w2, dtype, page, prefix="n.")
    if keep is None:
        own.keep = None
    cache = CacheManager([own.cache_needs()], page, 40, 3, dtype=DT[dtype], device=DEV)
    cache.open("other")

    def run(x, entries):
        ctx = context_for(cache, entries, own, reader)
        xd = dev(x, DT[dtype])
        return np.concatenate([summed(own.forward(xd, ctx, cache.views(0), True)),
                               summed(reader.forward(xd, ctx, cache.views(0), False))], axis=1)

    got = run_in_steps(run, cache, streams, STEPS)
    tol = 2e-4 if dtype == "float32" else 4e-2
    for r in streams:
        assert np.abs(got[r] - want[r]).max() < tol * max(1.0, np.abs(want[r]).max()), (r, float(np.abs(got[r] - want[r]).max()))
    if keep is not None and keep < 200:
        assert cache.used_pages("a") < 320 // page, "pages went back"
    cache.close("b")
    again = run_in_steps(run, cache, {"c": streams["b"]}, [[("c", 5)], [("c", 1)], [("c", 69)]])     # b's slot and pages
    assert np.abs(again["c"] - want["b"]).max() < tol * max(1.0, np.abs(want["b"]).max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,E,window", [(16, 128, 200), (64, 320, 200), (128, 640, 193), (16, 128, 17)])
def test_keys_just_inside_and_just_outside_the_window(d, E, window, dtype):
    """Keys and queries made by hand: two late queries point at the same key (a score that stands out among all others; the
    query is the key turned back by the distance), one from the last place that still sees it and one from the first that
    does not; the values show which key was found.  As one prompt, with decoded tokens, and in ragged portions, on
    scattered pages."""
    from air_b200.cache.manager import CacheManager
    H, G, dv, T, eps = 2, 1, d, 420, 1e-6
    m = du.attention(H, G, d, dv, 0.6, window, d // 2, 10000.0)["mixer"]
    rng = np.random.default_rng(7)
    w = attention_weights(rng, E, m, dtype)
    w["q.norm"], w["k.norm"], w["temp"] = np.full(d, 2.0), np.full(d, 2.0), np.array([1.0, 0.75])
    x = rng.normal(size=(T, E)) * 0.3
    last = {}                                          # query place -> the key it points at
    for j in (0, 15, 16, 63, 64, 128, 200):
        last[j + window - 1], last[j + window] = j, j
    last = {i: j for i, j in last.items() if i < T and i not in (0, 15, 16, 63, 64, 128, 200)}
    pos = np.arange(T)
    for i, j in last.items():
        key = plain.over_rms((x[j:j + 1] @ w["k"].T).reshape(1, G, d), eps) * w["k.norm"]
        back = plain.turn(plain.turn(key, [j], d // 2, 10000.0, np.float64), [-i], d // 2, 10000.0, np.float64)
        back = np.repeat(back, H, axis=1).reshape(-1)
        # Wq x[i] is that query, Wk x[i] is against it (its own key does not draw it), Wv x[i] is nothing
        x[i] = np.linalg.lstsq(np.concatenate([w["q"], w["k"], w["v"]]),
                               np.concatenate([back, -back[:G * d], np.zeros(G * dv)]), rcond=None)[0]
    if dtype == "bfloat16":
        x = du.bf16(x).astype(np.float64)
    wp = {"m." + k: a for k, a in w.items()}
    want, _ = plain.mixer_attention(wp, "m.", x, m, pos, eps, np.float64)
    # the window's edge shows: one token more or less moves the rows that stand at it
    for off in (-1, 1):
        moved, _ = plain.mixer_attention(wp, "m.", x, dict(m, mask=dict(size=window + off)), pos, eps, np.float64)
        edge = [i for i, j in last.items() if (i - j == window - 1) == (off < 0)]
        assert (np.abs(moved - want)[edge].max(axis=1) > 0.2 * np.abs(want).max()).mean() > 0.8
    part = load(attention_part(E, m, eps), w, dtype)
    for cuts in ([T], [380] + [1] * 40, [7, 9, 1, 383, 2, 2, 16], [window, 1, T - window - 1]):
        cache = CacheManager([part.cache_needs()], 16, 40, 2, dtype=DT[dtype], device=DEV)
        for g in cache.groups:              # pages in an order of their own
            rng.shuffle(g.pool._free)

        def run(rows, entries):
            ctx = context_for(cache, entries, part)
            return summed(part.forward(dev(rows, DT[dtype]), ctx, cache.views(0), True))

        got = run_in_steps(run, cache, {"r": x}, [[("r", n)] for n in cuts])["r"]
        tol = 2e-4 if dtype == "float32" else 4e-2
        assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), (cuts[:3], float(np.abs(got - want).max()))


def mlstm_weights(rng, E, H, d, dv, dtype):
    q = rng.normal(size=(H * d, E)) * 1.5 / E ** 0.5       # (keys near the queries: see dafotar_util.draw_tensors)
    w = {"q": q, "k": q + rng.normal(size=(H * d, E)) * 0.7 / E ** 0.5,
         "v": rng.normal(size=(H * dv, E)) * 1.5 / E ** 0.5, "g": rng.normal(size=(H * dv, E)) * 2 / E ** 0.5,
         "i": rng.normal(size=(H, E)) * 2.0 / E ** 0.5, "f": rng.normal(size=(H, E)) / E ** 0.5,
         "i.b": rng.normal(0.0, 1.5, size=H), "f.b": np.array([(12.0, -3.0, 3.0, 6.0)[h % 4] for h in range(H)]),
         "norm": rng.normal(1.0, 0.15, size=H * dv), "o": rng.normal(size=(E, H * dv)) / (H * dv) ** 0.5}
    return rounded(w, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,dv,cap", [(3, 20, 12, 5.0), (1, 24, 40, 30.0), (4, 8, 8, 3.0), (2, 64, 128, 15.0), (3, 10, 6, 6.0),
                                        (1, 70, 22, 20.0), (2, 136, 144, 15.0), (2, 32, 64, 9.0), (1, 1, 1, 4.0),
                                        (2, 130, 258, 25.0)])
def test_mlstm_carries_its_state_through_portions_and_slots(H, d, dv, cap, dtype):
    """The mixer alone: two requests in steps that hold both, portions of many sizes (chunks that are full, cut and single)
    and single tokens; a first token of thirty times the others' size and an input gate far above all others, which the heads
    that hardly forget still show 300 tokens later, while other heads forget everything in between; a slot that another
    request held starts from zeros."""
    from air_b200.cache.manager import CacheManager
    from air_b200.parts.recurrent import MLSTM
    from air_b200.parts.spec import PartSpec
    E, eps = 72, 1e-5
    rng = np.random.default_rng(H * d + dv)
    w = mlstm_weights(rng, E, H, d, dv, dtype)
    streams = {"a": rng.normal(size=(320, E)), "b": rng.normal(size=(75, E))}
    streams["a"][0] *= 30.0
    streams["a"][0] += 20.0 * (w["i"][0] / np.square(w["i"][0]).sum())
    if dtype == "bfloat16":
        streams = {r: du.bf16(x).astype(np.float64) for r, x in streams.items()}
    m = dict(heads=H, dim=d, vdim=dv, gate_cap=cap)
    wp = {"m." + k: a for k, a in w.items()}
    want = {r: plain.mixer_mlstm(wp, "m.", x, m, None, eps, np.float64)[0] for r, x in streams.items()}
    if cap >= 12:
        short = plain.mixer_mlstm(wp, "m.", streams["a"][1:], m, None, eps, np.float64)[0]
        assert np.abs(short[-1] - want["a"][-1]).max() > 0.02 * np.abs(want["a"][-1]).max()      # the first token still shows
    part = load(MLSTM(PartSpec("mlstm", {"hidden": E, "heads": H, "head_dim": d, "v_dim": dv, "gate_cap": cap, "eps": eps}),
                      "m."), w, dtype)
    tol = 3e-4 if dtype == "float32" else 4e-2
    for steps in (STEPS, [[("a", 320), ("b", 75)]], [[("a", 64), ("b", 65)], [("a", 192)], [("b", 10), ("a", 64)]]):
        cache = CacheManager([part.cache_needs()], 16, 40, 3, dtype=DT[dtype], device=DEV)
        cache.open("other")

        def run(x, entries):
            ctx = context_for(cache, entries, part)
            return summed(part.forward(dev(x, DT[dtype]), ctx, cache.views(0), True))

        got = run_in_steps(run, cache, streams, steps)
        for r in streams:
            err = np.abs(got[r] - want[r]).max()
            assert err < tol * max(1.0, np.abs(want[r]).max()), (r, len(steps), float(err))
        cache.close("a")
        again = run_in_steps(run, cache, {"c": streams["b"]}, [[("c", 5)], [("c", 1)], [("c", 69)]])     # a's slot
        assert np.abs(again["c"] - want["b"]).max() < tol * max(1.0, np.abs(want["b"]).max())


@pytest.mark.parametrize("dtype,d,dv", [("float32", 48, 96), ("float32", 70, 130), ("bfloat16", 48, 96), ("bfloat16", 72, 136),
                                        ("bfloat16", 128, 128), ("bfloat16", 8, 8), ("bfloat16", 136, 264)])
def test_matrix_memory_in_chunks_against_token_by_token(dtype, d, dv):
    """Both roads of the matrix memory from the same projections, the states they leave behind among the results: chunks of
    a portion against one token at a time, from a state that is not empty, for gates that hold for long, close at once
    and jump; portions of every length around a chunk's; on the CUDA cores and (16-bit projections) on the tensor cores,
    where 32-bit operands enter as two 16-bit numbers."""
    from air_b200.csrc import ops
    rng = np.random.default_rng(5)
    H, cap = 4, 12.0
    for counts in ([63, 64, 65], [16, 128, 129], [200, 17, 191]):
        L, T = len(counts), sum(counts)
        start = np.concatenate([[0], np.cumsum(counts)])
        cols, at = {}, 0
        for n, width in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
            cols[n], at = at, at + width
        x = rng.normal(size=(T, at))
        x[:, :H * d] += 0.7 * x[:, H * d:2 * H * d]          # (a query near its key: the denominator is clear of zero)
        cols["i"], cols["f"] = H, 0
        z = np.concatenate([rng.normal(size=(T, H)) * np.array([0.1, 5.0, 1.0, 12.0]) + np.array([9.0, 0.0, 4.0, 0.0]),
                            rng.normal(size=(T, H)) * 3.0], axis=1)
        S0, n0, m0 = rng.normal(size=(3, H, d, dv)), rng.normal(size=(3, H, d)), rng.normal(size=(3, H))
        ib, fb, w = rng.normal(size=H), rng.normal(size=H), rng.normal(1.0, 0.2, size=H * dv)
        chunks, portions = [], []
        for i, n in enumerate(counts):
            portions.append((start[i], n, (2, 0, 1)[i], len(chunks)))
            chunks += [(start[i] + a, min(64, n - a)) for a in range(0, n, 64)]
        pair = []
        for road in ("tokens", "chunks"):
            S, n_, m_ = dev(S0), dev(n0), dev(m0)
            y = torch.zeros((T, H * dv), dtype=torch.float32, device=DEV)
            args = (dev(x, DT[dtype]), dev(z), cols, dev(ib), dev(fb), dev(w), S, n_, m_, y)
            if road == "tokens":
                ops.mlstm_step(*args, i32(start), i32((2, 0, 1)), cap, d ** -0.5, 1e-6)
            else:
                ops.mlstm_portions(*args, torch.tensor(np.array(portions), dtype=torch.int32, device=DEV),
                                   torch.tensor(np.array(chunks), dtype=torch.int32, device=DEV), cap, d ** -0.5, 1e-6)
            pair.append([t.cpu().numpy() for t in (y, S, n_, m_)])
        for what, a, b in zip("ySnm", *pair):
            assert np.isfinite(b).all()
            tol = 5e-5 if what != "y" else 2e-4
            assert np.abs(a - b).max() < tol * np.abs(a).max(), (what, counts, float(np.abs(a - b).max() / np.abs(a).max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,F,T", [(72, 100, 11), (96, 40, 70), (128, 256, 150), (40, 8, 3), (90, 50, 65), (256, 384, 600),
                                   (128, 128, 20)])
def test_gated_feed_forward_with_the_rectifier(E, F, T, dtype):
    """Both tcgen05 products with the rectifier in their epilogue, and the library's product with the activation kernel."""
    from air_b200.parts.mlp import ReGLU
    from air_b200.parts.spec import PartSpec
    rng = np.random.default_rng(E + F)
    w = rounded({"gate": rng.normal(size=(F, E)) * 1.4 / E ** 0.5, "up": rng.normal(size=(F, E)) * 1.4 / E ** 0.5,
                 "down": rng.normal(size=(E, F)) / F ** 0.5}, dtype)
    x = rng.normal(size=(T, E))
    if dtype == "bfloat16":
        x = du.bf16(x).astype(np.float64)
    part = load(ReGLU(PartSpec("reglu", {"hidden": E, "intermediate": F}), "m."), w, dtype)
    got = summed(part.forward(dev(x, DT[dtype]), SimpleNamespace(residual=None)))
    want = plain.dense_ff({"m." + k: a for k, a in w.items()}, "m.", x)
    assert np.abs(got - want).max() < (1e-4 if dtype == "float32" else 4e-2) * max(1.0, np.abs(want).max())


# ----------------------------------------------------------------------------- whole models
LENGTHS = {"A": (1, 7, 33, 97, 150), "B": (5, 40, 131, 64), "C": (2, 65, 150, 300), "D": (3, 70, 1, 129),
           "E": (130, 2, 310)}


def streams_for(name, seed=0, lengths=None):
    return {f"{name}{i}": du.tokens_for(name, n, seed + i) for i, n in enumerate(lengths or LENGTHS[name])}


def replay(name, dtype, steps, page_tokens=16, max_requests=4, peak_page=64):
    return util.replay(du.model_folder(name), dtype, steps, max_tokens=util.peak_tokens(steps, page=peak_page),
                       page_tokens=page_tokens, max_requests=max_requests)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_the_streams_after_every_layer(name, dtype):
    """Layer by layer: the sum of the streams behind every layer against the plain implementation's, for a prompt."""
    from air_b200.engine.batch import Entry
    from air_b200.engine.engine import Engine, EngineConfig
    cfg, tensors = du.plain_model(name)
    toks = du.tokens_for(name, 90, 3)
    want = []
    plain.forward(cfg, tensors, toks, taps=want)
    engine = Engine.from_folder(du.model_folder(name), EngineConfig(dtype=dtype, page_tokens=16, max_tokens=256,
                                                                    max_requests=2))
    engine.model.tap = []
    engine.step([Entry("r", toks, [])])
    engine.check_status()
    assert len(engine.model.tap) == len(want) == len(engine.model.spec.order)
    for i, (a, b) in enumerate(zip(engine.model.tap, want)):
        tol = 1e-4 if dtype == "float32" else 0.05
        assert np.abs(a.cpu().numpy() - b).max() < tol * np.abs(b).max(), (i, float(np.abs(a.cpu().numpy() - b).max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_whole_prompts(name, dtype):
    streams = streams_for(name)
    got, _ = replay(name, dtype, util.trace_whole(streams))
    print(name, dtype, du.check(got, name, streams, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "E"])
def test_prompt_then_token_by_token(name, dtype):
    streams = streams_for(name, 10)
    got, _ = replay(name, dtype, util.trace_bulk_tail(streams, tail=75))
    du.check(got, name, streams, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_down_to_two_tokens(name, dtype):
    streams = streams_for(name, 20)
    got, _ = replay(name, dtype, util.trace_portions(streams))
    du.check(got, name, streams, dtype)
    got, _ = replay(name, dtype, util.trace_portions(streams, sizes=(2, 2, 1, 3, 16, 15, 17, 64, 63, 65, 2)), page_tokens=64)
    du.check(got, name, streams, dtype)


@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_unequal_requests_together_with_pages_and_slots_used_again(name, dtype, page):
    """Many requests through three slots and a pool that holds the peak only: every request must come out as it does
    alone (the oracle runs each alone), whatever shared its batches and whoever had its slot (the matrix memories, the
    convolutions' last inputs) and its pages before."""
    lengths = LENGTHS[name] + ((120, 2, 77, 101, 64, 129) if name != "E" else (77, 1, 64))
    streams = streams_for(name, 50, lengths)
    steps = util.trace_mixed(streams, seed=3, live=3)
    got, engine = replay(name, dtype, steps, page_tokens=page, max_requests=3)
    du.check(got, name, streams, dtype)
    for group in engine.cache.groups:
        assert group.pool.takes > group.pool.num_pages, "pages were used again"


@pytest.mark.parametrize("name", ["random1", "random2", "random3", "random5", "random8", "random13", "random21", "random34"])
def test_configurations_drawn_at_random(name):
    """Layer orders, sizes and constants that nobody chose (dafotar_util.random_config): whole prompts and a mixed schedule
    through three slots, in float32 within its tolerance; bfloat16 must be finite and agree with the oracle in the median
    (how far single rows lie depends on how a drawn model amplifies rounding)."""
    du.model_folder(name)
    streams = {f"{name}_{i}": du.tokens_for(name, n, 80 + i) for i, n in enumerate((150, 3, 70, 1, 97))}
    whole = util.trace_whole(streams)
    mixed = util.trace_mixed(streams, seed=5, live=3, tail=20)
    got, _ = replay(name, "float32", whole, page_tokens=64)
    du.check(got, name, streams, "float32")
    got, _ = replay(name, "float32", mixed, page_tokens=16, max_requests=3)
    du.check(got, name, streams, "float32")
    for steps, page in ((whole, 16), (mixed, 64)):
        got, _ = replay(name, "bfloat16", steps, page_tokens=page, max_requests=3)
        means = []
        for (rid, p), row in got.items():
            ref = du.plain_logits(name, streams[rid])
            assert np.isfinite(row).all()
            means.append(np.abs(row - ref[p]).mean() / max(1.0, np.abs(ref).max()))
        assert np.median(means) <= 2 * du.BF16_MEDIAN_TOL, (name, float(np.median(means)))


@pytest.mark.parametrize("name", ["A", "C"])
def test_float32_does_not_depend_on_the_cut_or_the_batch(name):
    streams = streams_for(name, 30, (97, 40, 131))
    whole, _ = replay(name, "float32", util.trace_whole(streams))
    cut, _ = replay(name, "float32", util.trace_portions(streams, sizes=(2, 31, 1, 16, 5)))
    mixed, _ = replay(name, "float32", util.trace_mixed(streams, seed=1, live=3), max_requests=3)
    for key, row in whole.items():
        assert np.abs(cut[key] - row).max() < 3e-5 * max(1.0, np.abs(row).max())
        assert np.abs(mixed[key] - row).max() < 3e-5 * max(1.0, np.abs(row).max())


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_bfloat16_agrees_with_itself_across_schedules(name):
    streams = streams_for(name, 30, (97, 40, 131))
    whole, _ = replay(name, "bfloat16", util.trace_whole(streams), page_tokens=64)
    cut, _ = replay(name, "bfloat16", util.trace_portions(streams, sizes=(2, 31, 1, 16, 5)), page_tokens=64)
    mixed, _ = replay(name, "bfloat16", util.trace_mixed(streams, seed=1, live=3), page_tokens=64, max_requests=3)
    for other in (cut, mixed):
        means = []
        for key, row in whole.items():
            scale = max(1.0, np.abs(row).max())
            diff = np.abs(other[key] - row)
            assert diff.max() <= 2 * du.BF16_MAX_TOL * scale and diff.mean() <= 2 * du.BF16_MEAN_TOL * scale, key
            means.append(diff.mean() / scale)
        assert np.median(means) <= du.BF16_MEDIAN_TOL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_page_borders_and_first_tokens(name, dtype):
    """Prompts that end just before, on and just behind a page's last place, then decoded across the border; and
    requests decoded from their very first token (the convolutions see zeros ahead of it, mlstm an empty memory)."""
    from air_b200.engine.batch import Entry
    from air_b200.engine.engine import Engine, EngineConfig
    engine = Engine.from_folder(du.model_folder(name), EngineConfig(dtype=dtype, page_tokens=16, max_tokens=1024,
                                                                    max_requests=4))
    for n in (15, 16, 17, 31, 33):
        toks = du.tokens_for(name, n + 4, n)
        got = [engine.step([Entry("r", toks[:n], range(n))]).cpu().numpy()]
        got += [engine.step([Entry("r", [t], [0])]).cpu().numpy() for t in toks[n:]]
        engine.finish("r")
        du.check({("r", p): row for p, row in enumerate(np.concatenate(got))}, name, {"r": toks}, dtype)
    toks = du.tokens_for(name, 6, 99)
    got = np.concatenate([engine.step([Entry("s", [t], [0])]).cpu().numpy() for t in toks])
    du.check({("s", p): row for p, row in enumerate(got)}, name, {"s": toks}, dtype)
    got = [engine.step([Entry("t", toks[:2], [0, 1])]).cpu().numpy()]
    got += [engine.step([Entry("t", [t], [0])]).cpu().numpy() for t in toks[2:]]
    du.check({("t", p): row for p, row in enumerate(np.concatenate(got))}, name, {"t": toks}, dtype)
    engine.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding(name, dtype):
    """320 tokens one by one after a prompt of five, across twenty pages (the decode steps replay a CUDA graph)."""
    from air_b200.engine.batch import Entry
    from air_b200.engine.engine import Engine, EngineConfig
    toks = du.tokens_for(name, 325, 7)
    engine = Engine.from_folder(du.model_folder(name), EngineConfig(dtype=dtype, page_tokens=16, max_tokens=384,
                                                                    max_requests=2))
    got = [engine.step([Entry("r", toks[:5], range(5))]).cpu().numpy()]
    got += [engine.step([Entry("r", [t], [0])]).cpu().numpy() for t in toks[5:]]
    du.check({("r", p): row for p, row in enumerate(np.concatenate(got))}, name, {"r": toks}, dtype)
    assert engine.graphs, "decode steps ran as a graph"
    engine.check_status()


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_service(name):
    """The scheduler cuts prompts into portions of five, decodes one step ahead and feeds the device's own choice back."""
    from air_b200 import GenerationConfig
    from air_b200.engine.engine import Engine, EngineConfig
    from air_b200.engine.service import InferenceService, SchedulerConfig
    engine = Engine.from_folder(du.model_folder(name), EngineConfig(dtype="float32", page_tokens=16, max_tokens=1024,
                                                                    max_requests=4))
    svc = InferenceService(engine, SchedulerConfig(max_active_requests=4, prefill_quantum_tokens=5,
                                                   token_budget_per_cycle=12))
    prompts = [du.tokens_for(name, n, 40 + n) for n in (1, 7, 33, 20, 3)]
    want = [du.plain_greedy(name, p, 12) for p in prompts]
    got = svc.generate_cohort([(p, GenerationConfig(max_new_tokens=12, stop_on_eos=False)) for p in prompts])
    assert [r.tokens for r in got] == want
    assert engine.cache.free_pages() == engine.cache.num_pages
    engine.check_status()


def test_trace_runner_program_and_command_line(capsys):
    """bin/trace_run as a program on a Dafotar folder (the class is chosen by config.json), and the command line."""
    name = "B"
    streams = streams_for(name, 60, (40, 9))
    steps = util.trace_mixed(streams, seed=2, live=2)
    with tempfile.TemporaryDirectory() as out:
        util.run_trace_program(du.model_folder(name), "float32", steps, util.peak_tokens(steps), out)
        got = util.collect(steps, out, du.CONFIGS[name]["vocab"])
    du.check(got, name, streams, "float32")
    from air_b200 import cli
    prompt = du.tokens_for(name, 9, 70)
    assert cli.main(["cuda", du.model_folder(name), ",".join(map(str, prompt)), "--tokens", "6", "--dtype", "float32",
                     "--no-stop-on-eos"]) == 0
    assert capsys.readouterr().out.strip() == ",".join(map(str, du.plain_greedy(name, prompt, 6)))
