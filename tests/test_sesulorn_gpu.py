"""Sesulorn on the GPU against the plain implementation (tests/plain/sesulorn_plain.py, 64-bit): every mechanism alone
through its part or kernel, then whole models through Engine.step, the scheduler and the trace runner, in float32 and
bfloat16, for configurations that differ in every size and option (sesulorn_util.CONFIGS)."""
import tempfile
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import sesulorn_util as su
import util
from plain import sesulorn_plain as plain

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
    return {k: su.bf16(a).astype(np.float64) for k, a in w.items()} if dtype == "bfloat16" else w


def load(part, w, dtype, page=16, prefix="m."):
    part.load({prefix + k: dev(a, DT[dtype]) for k, a in w.items()}, runtime(dtype, page))
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


def part_of(layer, E, eps, dtype, page=16, w=None, rng=None):
    """(the mixer as the registry builds it from the layer's configuration, its tensors)."""
    from air_b200.config import load_config
    from air_b200.parts import registry
    c = load_config(su.config(10, E, eps, None, [su.bare(layer)]))
    spec = registry.architecture("Sesulorn").build_spec(c).layers[0].parts["mixer"]
    w = rounded(w if w is not None else su.mixer_tensors(rng, E, layer), dtype)
    return load(registry.MIXERS.get(spec.kind)(spec, "m."), w, dtype, page), w


def mixer_against_plain(layer, E, eps, dtype, page, seed, tol, steps=STEPS, shuffle=False):
    """The mixer alone: two requests in steps that hold both, portions of many sizes and single tokens, against the plain
    function on each whole sequence; then a third request on the second one's slot and pages."""
    from air_b200.cache.manager import CacheManager
    rng = np.random.default_rng(seed)
    part, w = part_of(layer, E, eps, dtype, page, rng=rng)
    streams = {"a": rng.normal(size=(320, E)), "b": rng.normal(size=(75, E))}
    if dtype == "bfloat16":
        streams = {r: su.bf16(x).astype(np.float64) for r, x in streams.items()}
    wp = {"m." + k: a for k, a in w.items()}
    want = {r: plain.MIXERS[layer["type"]](wp, "m.", x, layer["mixer"], eps, np.float64) for r, x in streams.items()}
    cache = CacheManager([part.cache_needs()], page, 40, 3, dtype=DT[dtype], device=DEV)
    cache.open("other")

    def run(x, entries):
        ctx = context_for(cache, entries, part)
        y = summed(part.forward(dev(x, DT[dtype]), ctx, cache.views(0), True))
        assert int(ctx.status.item()) == 0
        return y

    got = run_in_steps(run, cache, streams, steps)
    for r in streams:
        err = np.abs(got[r] - want[r]).max()
        assert err < tol * max(1.0, np.abs(want[r]).max()), (r, float(err))
    cache.close("b")
    again = run_in_steps(run, cache, {"c": streams["b"]}, [[("c", 5)], [("c", 1)], [("c", 69)]])     # b's slot and pages
    assert np.abs(again["c"] - want["b"]).max() < tol * max(1.0, np.abs(want["b"]).max())
    return streams, want


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,parts", [(1, 72, (1, 1, 1)), (13, 90, (3, 2, 1)), (300, 256, (2, 4, 1)), (2, 2048, (4, 4, 4)),
                                       (700, 4160, (1, 2, 1)), (9, 10, (1, 1, 2))])
def test_sums_of_three_terms_norms_and_rows_beside_the_embedding(T, E, parts, dtype):
    """What a layer with a mixer, experts and a gated shared expert side by side hands on: the stream completed and
    normalised in one pass, for chosen rows, completed alone, and written beside the embedding's output as it is; with
    the layer norm and with the RMS norm."""
    from air_b200.csrc import ops
    from air_b200.parts.base import GatedSum, Norm, ScaledSum, row_terms
    from air_b200.parts.block import ParallelBlock
    from air_b200.parts.norm import LayerNorm, RMSNorm
    from air_b200.parts.spec import PartSpec
    rng = np.random.default_rng(T + E)
    eps = 1e-5
    w, b = rng.normal(1.0, 0.3, size=E), rng.normal(0.0, 0.5, size=E)
    ln = LayerNorm(PartSpec("layer", {"size": E, "eps": eps, "tensor": "", "bias": ".b"}), "n")
    ln.load({"n": dev(w), "n.b": dev(b)}, runtime(dtype))
    rms = RMSNorm(PartSpec("rms", {"size": E, "eps": eps, "tensor": ""}), "n")
    rms.load({"n": dev(w)}, runtime(dtype))
    tol = 2e-5 if dtype == "float32" else 2e-2
    h, x0 = rng.normal(size=(T, E)) * 3 + 4, rng.normal(size=(T, E))
    ys = [rng.normal(size=(n, T, E)) * 2 for n in parts]
    gate = rng.uniform(size=T)
    dy = [dev(y if len(y) > 1 else y[0]) for y in ys]
    delta = ScaledSum(ParallelBlock._terms(dy[0], None) + ParallelBlock._terms(GatedSum(dy[1], dy[2], dev(gate)), None))
    assert len(row_terms(delta)) == 3
    after = h + ys[0].sum(0) + ys[1].sum(0) + gate[:, None] * ys[2].sum(0)
    over = after / np.sqrt((after * after).mean(axis=1, keepdims=True) + eps) * w
    close = lambda a, want, t: np.abs(a.float().cpu().numpy() - want).max() < t * np.abs(want).max()
    pick = [T - 1, 0, T // 2]
    for norm, want in ((ln, plain.layer_norm(after, w, b, eps)), (rms, over)):
        hd = dev(h)
        assert close(norm.forward(hd, delta), want, tol) and close(hd, after, 2e-5)
        hd = dev(h)
        assert close(norm.forward(hd, delta, rows=i32(pick)), want[pick], tol) and close(hd, h, 1e-7)
    assert close(Norm.add_delta(dev(h), delta), after, 2e-5)
    terms = row_terms(delta)
    out = torch.empty((T, 2 * E), dtype=DT[dtype], device=DEV)
    ops.stream_norm(dev(h), 1, None, None, 0.0, out, term=terms[0][0], more=terms[1:], again=dev(x0))
    assert close(out[:, :E], after, tol) and close(out[:, E:], x0, tol)
    out = torch.empty((T, 2 * E), dtype=DT[dtype], device=DEV)
    ops.stream_norm(dev(h), 1, None, None, 0.0, out, again=dev(x0))
    assert close(out[:, :E], h, tol) and close(out[:, E:], x0, tol)


ATTENTION = [      # heads, kv_heads, dim, vdim, rows of the table, its reach, page
    (6, 2, 16, 20, 8, 40, 16),
    (4, 4, 8, 16, 2, 3, 16),
    (1, 1, 32, 24, 10, 6, 32),
    (3, 1, 14, 10, 14, 60, 16),
    (4, 2, 64, 64, 16, 300, 64),
    (4, 1, 128, 128, 32, 128, 32),
    (8, 2, 64, 64, 8, 20, 16),
    (20, 1, 64, 64, 32, 1000, 64),
    (2, 2, 32, 40, 32, 100, 16),
    (2, 1, 256, 256, 8, 70, 64),
    (18, 1, 64, 32, 32, 77, 16),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,rows,span,page", ATTENTION)
def test_attention_with_a_distance_bias(H, G, d, dv, rows, span, page, dtype):
    layer = su.attention(H, G, d, dv, 2.0 / d ** 0.5, rows, span)
    mixer_against_plain(layer, 80, 1e-5, dtype, page, H * d + dv, 2e-4 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,dv,page", [(64, 64, 64), (128, 128, 16), (16, 24, 16), (14, 10, 16), (256, 256, 64)])
@pytest.mark.parametrize("rows,span", [(16, 128), (8, 300), (6, 8)])
def test_every_row_of_the_distance_table_from_its_first_to_its_last_distance(rows, span, d, dv, page, dtype):
    """All scores are equal but for the bias, and every head's table has one row that stands out: its output is the mean of
    the values at exactly that row's distances.  The value of position j is a number of its own, so a row that begins or ends
    one position off shows, also at rows of one distance, at the last row (keys of any distance) and in the tiles where
    the table's reach ends.  As one prompt, with decoded tokens, and in ragged portions, on scattered pages."""
    from air_b200.cache.manager import CacheManager
    E, T, eps = 80, 420, 1e-6
    H = rows
    rng = np.random.default_rng(rows + d)
    layer = su.attention(H, 1, d, dv, 0.1, rows, span)
    w = su.mixer_tensors(rng, E, layer)
    for n in "qk":                # q and k are their biases: the same for every token
        w[n], w[n + ".b"] = np.zeros_like(w[n]), np.ones_like(w[n + ".b"])
    w["v.b"] = np.zeros(dv)
    w["rel"] = np.where(np.eye(rows) > 0, 14.0, 0.0)
    x = rng.normal(size=(T, E))
    part, w = part_of(layer, E, eps, dtype, page, w=w)
    x = su.bf16(x).astype(np.float64) if dtype == "bfloat16" else x
    wp = {"m." + k: a for k, a in w.items()}
    want = plain.mixer_attention(wp, "m.", x, layer["mixer"], eps, np.float64)
    # one distance more or less at any row's edge is seen
    spread = np.array([plain.bucket(n, rows, span) for n in range(T)])
    v = x @ w["v"].T
    for b in range(rows):
        back = np.nonzero(spread == b)[0]
        i = T - 1
        mean = v[i - back].mean(axis=0)
        for other in ([i - back[0] + 1] if back[0] else []) + ([i - back[-1] - 1] if back[-1] < T - 1 else []):
            assert np.abs(np.concatenate([v[i - back], v[other:other + 1]]).mean(axis=0) - mean).max() > 1.5 / (len(back) + 1)
    tol = 2e-4 if dtype == "float32" else 2e-2
    for cuts in ([T], [380] + [1] * 40, [7, 9, 1, 383, 2, 2, 16], [span.__int__(), 1, T - int(span) - 1]):
        cache = CacheManager([part.cache_needs()], page, 40, 2, dtype=DT[dtype], device=DEV)
        for g in cache.groups:              # pages in an order of their own
            rng.shuffle(g.pool._free)

        def run(rows_, entries):
            ctx = context_for(cache, entries, part)
            return summed(part.forward(dev(rows_, DT[dtype]), ctx, cache.views(0), True))

        got = run_in_steps(run, cache, {"r": x}, [[("r", n)] for n in cuts])["r"]
        assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), (cuts[:3], float(np.abs(got - want).max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["tiles", "narrow", "latent"])
def test_one_far_key_among_hundreds(kind, dtype):
    """A query that points at one key far back, at page borders and at the first tokens: its score stands out, and the
    output is that key's value.  For a distance table the last row is what such a key gets."""
    from air_b200.cache.manager import CacheManager
    E, T, eps = 640, 420, 1e-6
    rng = np.random.default_rng(5)
    if kind == "latent":
        layer = su.latent(2, 24, 8, 20, 40, 200, 0.3, 10000.0)
    else:
        layer = su.attention(2, 1, *((64, 64) if kind == "tiles" else (24, 16)), 0.35 if kind == "tiles" else 0.9, 8, 64)
    m = layer["mixer"]
    w = su.mixer_tensors(rng, E, layer)
    x = rng.normal(size=(T, E)) * 0.3
    far = {T - 1: 0, T - 2: 1, T - 3: 15, T - 4: 16, T - 5: 63, T - 6: 64, 300: 2, 299: 127, 210: 128}
    H, d = m["heads"], m["dim"]
    if kind == "latent":
        for i, j in far.items():
            c = plain.over_rms(x[j:j + 1] @ w["dkv"][:m["kv_rank"]].T, eps) * w["dkv.norm"]
            key = (c @ w["uk"].T).reshape(H, d)
            q = np.zeros((H, d + m["rot_dim"]))
            q[:, :d] = key
            cq = np.linalg.lstsq(w["uq"], q.reshape(-1), rcond=None)[0] / w["dq.norm"]
            cq /= np.sqrt((cq ** 2).mean())          # (the query's latent is normalised: only its direction is free)
            x[i] = np.linalg.lstsq(np.concatenate([w["dq"], w["dkv"]]),
                                   np.concatenate([cq, 0.05 * rng.normal(size=len(w["dkv"]))]), rcond=None)[0]
    else:
        w["q.b"], w["k.b"] = np.zeros(H * d), np.zeros(d)
        for i, j in far.items():
            key = x[j] @ w["k"].T
            x[i] = np.linalg.lstsq(np.concatenate([w["q"], w["k"]]), np.concatenate([np.tile(key, H), -key]), rcond=None)[0]
    part, w = part_of(layer, E, eps, dtype, 16, w=w)
    x = su.bf16(x).astype(np.float64) if dtype == "bfloat16" else x
    wp = {"m." + k: a for k, a in w.items()}
    f = plain.MIXERS[layer["type"]]
    want = f(wp, "m.", x, m, eps, np.float64)
    for i, j in far.items():                     # the key matters: with its token replaced, the row is another one
        y = x[:i + 1].copy()
        y[j] = x[(j + 37) % 200 + 3]
        assert np.abs(f(wp, "m.", y, m, eps, np.float64)[i] - want[i]).max() > 0.1 * np.abs(want[i]).max(), (i, j)
    tol = 2e-4 if dtype == "float32" else 4e-2
    for cuts in ([T], [T - 8] + [1] * 8, [7, 9, 1, 383, 2, 2, 16]):
        cache = CacheManager([part.cache_needs()], 16, 40, 2, dtype=DT[dtype], device=DEV)
        for g in cache.groups:
            rng.shuffle(g.pool._free)

        def run(rows, entries):
            ctx = context_for(cache, entries, part)
            return summed(part.forward(dev(rows, DT[dtype]), ctx, cache.views(0), True))

        got = run_in_steps(run, cache, {"r": x}, [[("r", n)] for n in cuts])["r"]
        assert np.abs(got - want).max() < tol * max(1.0, np.abs(want).max()), (cuts[:3], float(np.abs(got - want).max()))


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 20), (1, 1, 64, 33), (2, 2, 130, 8), (3, 1, 16, 128), (2, 1, 600, 5),
                                      (1, 1, 1, 1)])
def test_channel_delta_scan(H, G, d, dv):
    """Against the plain recurrence: whole, and cut into portions of 1, 2, 17 and the rest (the state is carried), two
    requests in the batch, key sizes that are no powers of two and a value size that fills no block; channels that keep
    everything beside channels that forget at once."""
    from air_b200.csrc import ops
    rng = np.random.default_rng(d)
    T = 70
    a_log, dt_bias = rng.uniform(-2, 0.5, size=H), rng.choice([-9.0, -2.0, 1.0, 6.0], size=H * d)
    seqs, want = {}, {}
    for r in range(2):
        q, k, v = rng.normal(size=(T, G * d)), rng.normal(size=(T, G * d)), rng.normal(size=(T, H * dv))
        z, b = rng.normal(size=(T, H * d)) * 2, rng.normal(size=(T, H)) * 2
        seqs[r] = (q, k, v, z, b)
        g = np.exp(-np.exp(a_log)[:, None] * plain.softplus(z + dt_bias).reshape(T, H, d))
        want[r] = plain.delta_memory(plain.unit(q.reshape(T, G, d)) * d ** -0.5, plain.unit(k.reshape(T, G, d)),
                                     v.reshape(T, H, dv), g, plain.sigmoid(b), np.float64)
    for cuts in ([T], [1, 2, 17, T - 20]):
        state = torch.zeros((2, H, d, dv), device=DEV)
        at = 0
        for n in cuts:
            rows = [np.concatenate([seqs[r][i][at:at + n] for r in (1, 0)]) for i in range(5)]
            out = torch.empty((2 * n, H, dv), device=DEV)
            ops.linear_scan(ops.SCAN_CHANNEL_DELTA, dev(rows[0]), dev(rows[1]), dev(rows[2]), dev(rows[3]), state, out,
                            i32([0, n, 2 * n]), i32([1, 0]), i32([1] * n + [0] * n), q_scale=d ** -0.5, beta=dev(rows[4]),
                            a_log=dev(a_log), dt_bias=dev(dt_bias), unit=True)
            out = out.cpu().numpy()
            for j, r in enumerate((1, 0)):
                assert np.abs(out[j * n:(j + 1) * n] - want[r][at:at + n]).max() < 3e-5
            at += n


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 20), (1, 1, 64, 33), (2, 2, 130, 8), (3, 1, 16, 128), (2, 1, 256, 5), (1, 1, 1, 1),
                                      (2, 2, 128, 128), (6, 3, 12, 18)])
@pytest.mark.parametrize("decays", ["mixed", "slow", "fast"])
def test_delta_rule_in_chunks_against_token_by_token(decays, H, G, d, dv):
    """Both roads of the channel-wise delta rule and the plain recurrence, from states that are not empty, the states they
    leave behind among the results: portions of every length around a chunk's in one batch, channels that keep everything,
    that forget at once, and that change from one to the other from token to token; keys that repeat."""
    from air_b200.csrc import ops
    rng = np.random.default_rng(d + dv)
    for counts in ([15, 16, 17], [1, 32, 200], [48, 31, 2]):
        T = sum(counts)
        start = np.concatenate([[0], np.cumsum(counts)])
        a_log = rng.uniform(-2, 0.5, size=H)
        dt = {"mixed": rng.choice([-9.0, -2.0, 1.0, 6.0], size=H * d), "slow": np.full(H * d, -8.0), "fast": np.full(H * d, 9.0)}[decays]
        q, k, v = rng.normal(size=(T, G * d)), rng.normal(size=(T, G * d)), rng.normal(size=(T, H * dv))
        k[T // 3:T // 3 + 6] = k[T // 3]                 # the same key several times
        z, b = rng.normal(size=(T, H * d)) * 2, rng.normal(size=(T, H)) * 3
        z[::5] += 30.0 * (rng.random(size=(len(z[::5]), H * d)) < 0.2)
        S0 = rng.normal(size=(4, H, d, dv))
        slots = [2, 0, 3]
        chunks, portions = [], []
        for i, n in enumerate(counts):
            portions.append((start[i], n, slots[i], len(chunks)))
            chunks += [(start[i] + a, min(ops.DELTA_CHUNK, n - a)) for a in range(0, n, ops.DELTA_CHUNK)]
        wide = dev(np.concatenate([q, k, v], axis=1))          # bands of a wider matrix
        bands = (wide[:, :G * d], wide[:, G * d:2 * G * d], wide[:, 2 * G * d:], dev(z))
        kw = dict(q_scale=d ** -0.5, beta=dev(b), a_log=dev(a_log), dt_bias=dev(dt))
        got = []
        for road in ("tokens", "chunks"):
            S, o = dev(S0), torch.full((T, H, dv), 9.0, device=DEV)
            if road == "tokens":
                ops.linear_scan(ops.SCAN_CHANNEL_DELTA, *bands, S, o, i32(start), i32(slots),
                                i32(np.repeat(slots, counts)), unit=True, **kw)
            else:
                ops.delta_portions(*bands, S, o, torch.tensor(np.array(portions), dtype=torch.int32, device=DEV),
                                   torch.tensor(np.array(chunks), dtype=torch.int32, device=DEV), **kw)
            got.append((o.cpu().numpy(), S.cpu().numpy()))
        assert np.array_equal(got[1][1][1], S0[1].astype(np.float32)), "another request's state is not touched"
        g = np.exp(-np.exp(a_log)[:, None] * plain.softplus(z + dt).reshape(T, H, d))
        kk, qq = plain.unit(k.reshape(T, G, d)), plain.unit(q.reshape(T, G, d)) * d ** -0.5
        for i, n in enumerate(counts):
            for h in range(H):
                S = S0[slots[i], h].copy()
                for t in range(start[i], start[i] + n):
                    S = g[t, h][:, None] * S
                    S = S + np.outer(kk[t, h // (H // G)], plain.sigmoid(b[t, h]) * (v[t, h * dv:(h + 1) * dv] - S.T @ kk[t, h // (H // G)]))
                    for road in range(2):
                        assert np.abs(got[road][0][t, h] - S.T @ qq[t, h // (H // G)]).max() < 5e-5, (road, i, t)
                for road in range(2):
                    assert np.abs(got[road][1][slots[i], h] - S).max() < 5e-5 * max(1.0, np.abs(S).max()), (road, i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,taps,ra,rg", [(4, 2, 20, 12, 4, 6, 10), (1, 1, 24, 40, 1, 1, 1), (3, 1, 10, 6, 6, 3, 7),
                                                 (2, 2, 64, 64, 3, 16, 8), (2, 1, 136, 72, 2, 32, 40), (6, 3, 8, 8, 16, 5, 2),
                                                 (2, 2, 128, 128, 4, 64, 128)])
def test_channel_delta_carries_its_state_through_portions_and_slots(H, G, d, dv, taps, ra, rg, dtype):
    layer = su.delta(H, G, d, dv, taps, ra, rg)
    streams, want = mixer_against_plain(layer, 72, 1e-5, dtype, 16, H * d + dv, 3e-4 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_channel_delta_remembers_its_first_token(dtype):
    """A first token of thirty times the others' size, in heads whose slow channels hardly forget: 319 tokens later the
    output still shows it, through every cut."""
    from air_b200.cache.manager import CacheManager
    E, eps, T = 72, 1e-5, 320
    layer = su.delta(2, 1, 24, 16, 3, 6, 5)
    rng = np.random.default_rng(11)
    w = su.mixer_tensors(rng, E, layer)
    w["dt_bias"], w["A_log"], w["a2"] = np.full(48, -9.0), np.full(2, -1.0), w["a2"] * 0.2
    w["b"] *= 0.0                            # (half of every value is written)
    part, w = part_of(layer, E, eps, dtype, 16, w=w)
    x = rng.normal(size=(T, E))
    x[0] *= 30.0
    # the tokens behind it come back to its key only at the end
    key = np.concatenate([w["k"], w["q"]])
    null = np.eye(E) - np.linalg.pinv(key) @ key
    x[1:-1] = x[1:-1] @ null + 0.05 * x[1:-1]
    x[-1] = x[0] / 30.0
    x = su.bf16(x).astype(np.float64) if dtype == "bfloat16" else x
    wp = {"m." + k: a for k, a in w.items()}
    want = plain.mixer_channel_delta(wp, "m.", x, layer["mixer"], eps, np.float64)
    other = x.copy()
    other[0] *= -1.0
    assert np.abs(plain.mixer_channel_delta(wp, "m.", other, layer["mixer"], eps, np.float64)[-1] - want[-1]).max() > \
        0.05 * np.abs(want[-1]).max()
    tol = 3e-4 if dtype == "float32" else 4e-2
    for cuts in ([T], [1, 2, 17, 100, 199, 1], [64] * 5):
        cache = CacheManager([part.cache_needs()], 16, 40, 2, dtype=DT[dtype], device=DEV)

        def run(rows, entries):
            ctx = context_for(cache, entries, part)
            return summed(part.forward(dev(rows, DT[dtype]), ctx, cache.views(0), True))

        got = run_in_steps(run, cache, {"r": x}, [[("r", n)] for n in cuts])["r"]
        assert np.abs(got[[0, -1]] - want[[0, -1]]).max() < tol * max(1.0, np.abs(want[-1]).max()), cuts[:3]


def test_gate_behind_the_read_out_is_the_sigmoid():
    from air_b200.csrc import ops
    rng = np.random.default_rng(5)
    for T, H, dv in ((13, 3, 20), (7, 2, 33), (5, 4, 128)):
        o, gate, w = rng.normal(size=(T, H, dv)), rng.normal(size=(T, H * dv)) * 4, rng.normal(1, 0.1, size=dv)
        out = torch.empty((T, H * dv), device=DEV)
        ops.gated_rmsnorm(dev(o), dev(gate), dev(w), 1e-5, out, i32([0] * T), sigmoid=True)
        want = (plain.over_rms(o, 1e-5) * w).reshape(T, H * dv) * plain.sigmoid(gate)
        assert np.abs(out.cpu().numpy() - want).max() < 1e-5


def test_bands_split_into_two_halves():
    from air_b200.csrc import ops
    rng = np.random.default_rng(6)
    x = rng.normal(size=(9, 40)) * np.array([10.0 ** (i % 7 - 3) for i in range(40)])
    for at, a, b in ((3, 12, 20), (0, 4, 4), (8, 1, 31)):
        xa, xb = ops.split_bands(dev(x)[:, at:at + a + b], a, b)
        for got, want in ((xa, x[:, at:at + a]), (xb, x[:, at + a:at + a + b])):
            got, n = got.float().cpu().numpy().astype(np.float64), want.shape[1]
            assert np.abs(got[:, :n] + got[:, n:] - want).max() <= 2e-5 * np.abs(want).max()
            assert (np.abs(got[:, :n] + got[:, n:] - want) <= 2.0 ** -15 * np.abs(want)).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,rot,dv,R,Q", [(3, 24, 8, 20, 40, 28), (2, 16, 0, 24, 32, 16), (1, 8, 16, 40, 24, 40),
                                            (3, 10, 6, 14, 22, 18), (8, 32, 32, 32, 128, 64), (4, 64, 64, 64, 512, 256),
                                            (2, 12, 2, 9, 7, 5)])
def test_latent_attention_with_a_query_latent_and_neighbouring_pairs(H, d, rot, dv, R, Q, dtype):
    layer = su.latent(H, d, rot, dv, R, Q, 0.3, 700.0)
    mixer_against_plain(layer, 80, 1e-4, dtype, 16, H * d + dv, 2e-4 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("n,groups,keep,top", [(12, 4, 2, 3), (6, 3, 1, 2), (8, 8, 3, 2), (64, 8, 4, 6), (10, 1, 1, 4), (96, 32, 5, 7)])
def test_router_with_groups_marked_by_their_best_expert(n, groups, keep, top):
    from air_b200.csrc import ops
    rng = np.random.default_rng(n + top)
    T = 200
    z = rng.normal(size=(T, n + 1)) * 2
    expert, weight = torch.empty((T, top), dtype=torch.int32, device=DEV), torch.empty((T, top), device=DEV)
    gate = torch.empty(T, device=DEV)
    ops.moe_route(dev(z), n, top, expert, weight, gate, has_gate=True, score="softmax", groups=groups, keep=keep, mark="best")
    s = plain.softmax_rows(z[:, :n])
    want = [plain.chosen_experts(s[t], groups, keep, top) for t in range(T)]
    assert expert.cpu().numpy().tolist() == want
    assert np.abs(weight.cpu().numpy() - np.take_along_axis(s, np.array(want), axis=1)).max() < 1e-6
    assert np.abs(gate.cpu().numpy() - plain.sigmoid(z[:, n])).max() < 1e-6
    if 1 < keep < groups and n // groups > 1:      # the two marks choose differently
        ops.moe_route(dev(z), n, top, expert, weight, None, score="softmax", groups=groups, keep=keep)
        assert expert.cpu().numpy().tolist() != want


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,F,n,top,groups,shared,T", [(72, 40, 6, 3, (3, 2), 48, 11), (64, 32, 4, 4, None, 0, 70),
                                                       (128, 64, 8, 5, (8, 5), 128, 150), (90, 30, 6, 2, (2, 2), 22, 9),
                                                       (64, 64, 4, 2, (2, 1), 64, 400), (40, 24, 1, 1, None, 16, 3)])
def test_clamped_experts_beside_a_gated_shared_expert(E, F, n, top, groups, shared, T, dtype):
    """Both roads of the experts (400 rows over four experts are the library's), limits that cut on every side, another
    limit for the shared expert."""
    from air_b200.config import load_config
    from air_b200.parts import registry
    from air_b200.parts.base import GatedSum
    rng = np.random.default_rng(E + F)
    layer = su.moe(su.attention(1, 1, 8, 8, 0.3, 2, 3), n, top, F, 0.9, groups, shared or None, 0.5)
    c = load_config(su.config(10, E, 1e-5, None, [layer]))
    spec = registry.architecture("Sesulorn").build_spec(c).layers[0].parts["feed_forward"]
    mat = lambda o, i, g=1.0: rng.normal(0.0, g / np.sqrt(i), size=(o, i))
    w = {"router": mat(n, E, 2.0)}
    for e in range(n):
        w.update({f"e{e}.gate": mat(F, E, 1.5), f"e{e}.up": mat(F, E, 1.5), f"e{e}.down": mat(E, F)})
    if shared:
        w.update({"shared.gate": mat(shared, E, 1.5), "shared.up": mat(shared, E, 1.5), "shared.down": mat(E, shared),
                  "shared.sg": mat(1, E, 2.0)})
    w = rounded(w, dtype)
    part = load(registry.FEED_FORWARDS.get(spec.kind)(spec, "m."), w, dtype)
    x = rng.normal(size=(T, E))
    x = su.bf16(x).astype(np.float64) if dtype == "bfloat16" else x
    s = plain.softmax_rows(x @ w["router"].T)
    clear = []                               # rows whose choice no rounding changes
    for t in range(T):
        g, k = groups or (1, 1)
        chosen = plain.chosen_experts(s[t], g, k, top)
        jitter = [plain.chosen_experts(s[t] * (1 + 0.02 * rng.normal(size=n)), g, k, top) for _ in range(8)]
        if all(sorted(j) == sorted(chosen) for j in jitter):
            clear.append(t)
    assert len(clear) > T // 3
    y = part.forward(dev(x, DT[dtype]), SimpleNamespace(residual=None))
    if isinstance(y, GatedSum):
        got = summed(y.a) + y.gate.cpu().numpy()[:, None] * summed(y.b)
    else:
        got = summed(y)
    want = plain.moe_ff({"m." + k: a for k, a in w.items()}, "m.", x, layer["mlp"], np.float64)
    assert np.abs(got - want)[clear].max() < (1e-4 if dtype == "float32" else 3e-2) * max(1.0, np.abs(want).max())


# ----------------------------------------------------------------------------- whole models
LENGTHS = {"A": (1, 7, 33, 97, 150), "B": (5, 40, 131, 64), "C": (2, 65, 150, 300), "D": (3, 70, 1, 129),
           "E": (130, 2, 310)}


def streams_for(name, seed=0, lengths=None):
    return {f"{name}{i}": su.tokens_for(name, n, seed + i) for i, n in enumerate(lengths or LENGTHS[name])}


def replay(name, dtype, steps, page_tokens=16, max_requests=4, peak_page=64):
    return util.replay(su.model_folder(name), dtype, steps, max_tokens=util.peak_tokens(steps, page=peak_page),
                       page_tokens=page_tokens, max_requests=max_requests)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_the_stream_after_every_layer_run(name, dtype):
    """Layer by layer, every pass of a repeated stretch for itself, for a prompt and for a few rows (whose products leave
    partial sums)."""
    from air_b200.engine.batch import Entry
    from air_b200.engine.engine import Engine, EngineConfig
    cfg, tensors = su.plain_model(name)
    for n in (90, 20):
        toks = su.tokens_for(name, n, 3)
        want = []
        plain.forward(cfg, tensors, toks, taps=want)
        engine = Engine.from_folder(su.model_folder(name), EngineConfig(dtype=dtype, page_tokens=16, max_tokens=256,
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
    print(name, dtype, su.check(got, name, streams, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "E"])
def test_prompt_then_token_by_token(name, dtype):
    streams = streams_for(name, 10)
    got, _ = replay(name, dtype, util.trace_bulk_tail(streams, tail=75))
    su.check(got, name, streams, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_down_to_two_tokens(name, dtype):
    streams = streams_for(name, 20)
    got, _ = replay(name, dtype, util.trace_portions(streams))
    su.check(got, name, streams, dtype)
    got, _ = replay(name, dtype, util.trace_portions(streams, sizes=(2, 2, 1, 3, 16, 15, 17, 64, 63, 65, 2)), page_tokens=64)
    su.check(got, name, streams, dtype)


@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_unequal_requests_together_with_pages_and_slots_used_again(name, dtype, page):
    """Many requests through three slots and a pool that holds the peak only: every request must come out as it does
    alone (the oracle runs each alone), whatever shared its batches and whoever had its slot (matrix states, the
    convolutions' last inputs, a set for every pass) and its pages before."""
    lengths = LENGTHS[name] + ((120, 2, 77, 101, 64, 129) if name != "E" else (77, 1, 64))
    streams = streams_for(name, 50, lengths)
    steps = util.trace_mixed(streams, seed=3, live=3)
    got, engine = replay(name, dtype, steps, page_tokens=page, max_requests=3)
    su.check(got, name, streams, dtype)
    for group in engine.cache.groups:
        assert group.pool.takes > group.pool.num_pages, "pages were used again"


@pytest.mark.parametrize("name", ["random1", "random2", "random3", "random5", "random8", "random13", "random21", "random34",
                                  "random55"])
def test_configurations_drawn_at_random(name):
    """Layer orders, sizes and constants that nobody chose (sesulorn_util.random_config): whole prompts and a mixed schedule
    through three slots, in float32 within its tolerance; bfloat16 must be finite and agree with the oracle in the median
    (how far single rows lie depends on how a drawn model amplifies rounding)."""
    su.model_folder(name)
    streams = {f"{name}_{i}": su.tokens_for(name, n, 80 + i) for i, n in enumerate((150, 3, 70, 1, 97))}
    whole = util.trace_whole(streams)
    mixed = util.trace_mixed(streams, seed=5, live=3, tail=20)
    got, _ = replay(name, "float32", whole, page_tokens=64)
    su.check(got, name, streams, "float32")
    got, _ = replay(name, "float32", mixed, page_tokens=16, max_requests=3)
    su.check(got, name, streams, "float32")
    for steps, page in ((whole, 16), (mixed, 64)):
        got, _ = replay(name, "bfloat16", steps, page_tokens=page, max_requests=3)
        means = []
        for (rid, p), row in got.items():
            ref = su.plain_logits(name, streams[rid])
            assert np.isfinite(row).all()
            means.append(np.abs(row - ref[p]).mean() / max(1.0, np.abs(ref).max()))
        assert np.median(means) <= 2 * su.BF16_MEDIAN_TOL, (name, float(np.median(means)))


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
            assert diff.max() <= 2 * su.BF16_MAX_TOL * scale and diff.mean() <= 2 * su.BF16_MEAN_TOL * scale, key
            means.append(diff.mean() / scale)
        assert np.median(means) <= su.BF16_MEDIAN_TOL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_page_borders_and_first_tokens(name, dtype):
    """Prompts that end just before, on and just behind a page's last place, then decoded across the border; and
    requests decoded from their very first token (the convolutions see zeros ahead of it, the state heads nothing)."""
    from air_b200.engine.batch import Entry
    from air_b200.engine.engine import Engine, EngineConfig
    engine = Engine.from_folder(su.model_folder(name), EngineConfig(dtype=dtype, page_tokens=16, max_tokens=1024,
                                                                    max_requests=4))
    for n in (15, 16, 17, 31, 33):
        toks = su.tokens_for(name, n + 4, n)
        got = [engine.step([Entry("r", toks[:n], range(n))]).cpu().numpy()]
        got += [engine.step([Entry("r", [t], [0])]).cpu().numpy() for t in toks[n:]]
        engine.finish("r")
        su.check({("r", p): row for p, row in enumerate(np.concatenate(got))}, name, {"r": toks}, dtype)
    toks = su.tokens_for(name, 6, 99)
    got = np.concatenate([engine.step([Entry("s", [t], [0])]).cpu().numpy() for t in toks])
    su.check({("s", p): row for p, row in enumerate(got)}, name, {"s": toks}, dtype)
    got = [engine.step([Entry("t", toks[:2], [0, 1])]).cpu().numpy()]
    got += [engine.step([Entry("t", [t], [0])]).cpu().numpy() for t in toks[2:]]
    su.check({("t", p): row for p, row in enumerate(np.concatenate(got))}, name, {"t": toks}, dtype)
    engine.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(name, dtype):
    """320 tokens one by one after a prompt of five, across twenty pages (the decode steps replay a CUDA graph)."""
    from air_b200.engine.batch import Entry
    from air_b200.engine.engine import Engine, EngineConfig
    toks = su.tokens_for(name, 325, 7)
    engine = Engine.from_folder(su.model_folder(name), EngineConfig(dtype=dtype, page_tokens=16, max_tokens=384,
                                                                    max_requests=2))
    got = [engine.step([Entry("r", toks[:5], range(5))]).cpu().numpy()]
    got += [engine.step([Entry("r", [t], [0])]).cpu().numpy() for t in toks[5:]]
    su.check({("r", p): row for p, row in enumerate(np.concatenate(got))}, name, {"r": toks}, dtype)
    assert engine.graphs, "decode steps ran as a graph"
    engine.check_status()


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_service(name):
    """The scheduler cuts prompts into portions of five, decodes one step ahead and feeds the device's own choice back."""
    from air_b200 import GenerationConfig
    from air_b200.engine.engine import Engine, EngineConfig
    from air_b200.engine.service import InferenceService, SchedulerConfig
    engine = Engine.from_folder(su.model_folder(name), EngineConfig(dtype="float32", page_tokens=16, max_tokens=1024,
                                                                    max_requests=4))
    svc = InferenceService(engine, SchedulerConfig(max_active_requests=4, prefill_quantum_tokens=5,
                                                   token_budget_per_cycle=12))
    prompts = [su.tokens_for(name, n, 40 + n) for n in (1, 7, 33, 20, 3)]
    want = [su.plain_greedy(name, p, 12) for p in prompts]
    got = svc.generate_cohort([(p, GenerationConfig(max_new_tokens=12, stop_on_eos=False)) for p in prompts])
    assert [r.tokens for r in got] == want
    assert engine.cache.free_pages() == engine.cache.num_pages
    engine.check_status()


def test_trace_runner_program_and_command_line(capsys):
    """bin/trace_run as a program on a Sesulorn folder (the class is chosen by config.json), and the command line."""
    name = "B"
    streams = streams_for(name, 60, (40, 9))
    steps = util.trace_mixed(streams, seed=2, live=2)
    with tempfile.TemporaryDirectory() as out:
        util.run_trace_program(su.model_folder(name), "float32", steps, util.peak_tokens(steps), out)
        got = util.collect(steps, out, su.CONFIGS[name]["vocab"])
    su.check(got, name, streams, "float32")
    from air_b200 import cli
    prompt = su.tokens_for(name, 9, 70)
    assert cli.main(["cuda", su.model_folder(name), ",".join(map(str, prompt)), "--tokens", "6", "--dtype", "float32",
                     "--no-stop-on-eos"]) == 0
    assert capsys.readouterr().out.strip() == ",".join(map(str, su.plain_greedy(name, prompt, 6)))
