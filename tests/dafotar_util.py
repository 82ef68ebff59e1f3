"""Set-up of the Dafotar tests: small configurations that differ in every size and option, model folders with weights
drawn so that a fault shows, and the comparison with the plain implementation."""
import functools
import tempfile

import numpy as np

from bivizen_util import bf16


def attention(heads, kv_heads, dim, vdim, scale, window, dims, base, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if window is not None:
        m["mask"] = dict(size=window)
    if base:
        m["rot"] = dict(base=base, dims=dims)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m)


def mlstm(heads, dim, vdim, cap):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap))


def dense(layer, ff):
    return dict(layer, mlp=dict(kind="dense", ff=ff))


def bare(layer):
    return dict(layer, mlp=None)


def config(vocab, width, eps, streams, taps, layers):
    return dict(architecture="Dafotar", vocab=vocab, width=width, norm=dict(eps=eps), streams=streams,
                canon=dict(taps=taps), layers=layers)


# A: three layers read the keys and values of layer 0, one with a wider window than layer 0's own, one with a narrower;
#    values larger than keys; part of a head rotated; four taps; two streams; the last layer has no feed-forward.
# B: one stream, one tap (no state), one head; a window of one token and a window that no test prompt fills; a layer that
#    borrows from a layer that borrows nothing in between mlstm layers; as many key/value heads as query heads.
# C: four streams; heads of 64 with keys and values of one size (the dense decoder's tile kernels), windows at and around
#    a tile's size; mlstm with wide values; feed-forwards of whole blocks of 128 (the activation in the product's epilogue).
# D: no size is a multiple of 4 (the kernels' roads of one element per access); five streams; six taps; the norm's eps large.
# E: heads of 128, one key/value head, the whole head rotated; mlstm heads of more than 128 channels of v and more than 64
#    of k; three streams; a layer that rotates values but neither queries nor keys, and one without a window.
CONFIGS = {
    "A": config(211, 72, 1e-5, 2, 4, [
        dense(attention(6, 2, 16, 20, 0.3, 24, 8, 500.0), 100),
        dense(mlstm(3, 20, 12, 5.0), 40),
        bare(attention(6, 2, 16, 20, 0.2, 50, 8, 500.0, kv_from=0)),
        dense(attention(6, 2, 16, 20, 0.25, 7, 8, 500.0, kv_from=0), 56),
        bare(mlstm(2, 32, 24, 15.0))]),
    "B": config(150, 64, 1e-6, 1, 1, [
        bare(mlstm(1, 24, 40, 8.0)),
        dense(attention(1, 1, 32, 24, 0.2, 1, 32, 10000.0), 96),
        dense(attention(4, 4, 8, 16, 0.4, 1000, 4, 100.0), 64),
        bare(mlstm(4, 8, 8, 3.0)),
        dense(attention(4, 4, 8, 16, 0.4, 33, 4, 100.0, kv_from=2), 32)]),
    "C": config(190, 128, 1e-6, 4, 2, [
        dense(attention(4, 2, 64, 64, 0.125, 64, 32, 10000.0), 256),
        dense(mlstm(2, 64, 128, 15.0), 128),
        dense(attention(4, 2, 64, 64, 0.15, 130, 32, 10000.0, kv_from=0), 384),
        bare(mlstm(4, 32, 32, 10.0))]),
    "D": config(133, 90, 1e-3, 5, 6, [
        dense(mlstm(3, 10, 6, 6.0), 50),
        dense(attention(3, 1, 14, 10, 0.3, 17, 6, 1000.0), 34),
        bare(attention(3, 1, 14, 10, 0.3, 16, 6, 1000.0, kv_from=1)),
        dense(mlstm(1, 70, 22, 9.0), 30)]),
    "E": config(300, 256, 1e-6, 3, 3, [
        dense(attention(4, 1, 128, 128, 0.09, 100, 128, 1000000.0), 320),
        dense(mlstm(2, 136, 144, 15.0), 256),
        bare(attention(8, 4, 32, 32, 0.2, 48, 0, 10000.0)),
        dense(attention(2, 2, 32, 40, 0.2, None, 16, 10000.0), 128)]),
}
SEEDS = {"A": 51, "B": 52, "C": 53, "D": 54, "E": 55}


def random_config(seed):
    """A configuration drawn at random: 2 to 6 layers in any order, every size and constant from a list that includes 1,
    equal and unequal sizes and sizes that are no multiples of 8 or 16; some attention layers read an earlier one's keys."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers, owners = [], []
    for i in range(int(rng.integers(2, 7))):
        if rng.random() < 0.6:
            if owners and rng.random() < 0.5:
                j = owners[int(rng.integers(len(owners)))]
                o = layers[j]["mixer"]
                r = o.get("rot", {})
                layer = attention(o["heads"], o["kv_heads"], o["dim"], o["vdim"], pick(0.1, 0.2, 0.3),
                                  pick(1, 5, 16, 17, 40, 64, 200), r.get("dims", 0), r.get("base", 0), kv_from=j)
            else:
                dim = pick(8, 16, 24, 32, 64)
                kv = pick(1, 2, 3)
                layer = attention(kv * pick(1, 2, 4), kv, dim, pick(8, 16, 24, 40, 64, dim), pick(0.1, 0.2, 0.3),
                                  pick(1, 5, 16, 17, 40, 64, 200), pick(0, 2, 4, 8, dim), pick(100.0, 10000.0, 500000.0))
                owners.append(i)
        else:
            layer = mlstm(pick(1, 2, 3, 4), pick(4, 8, 20, 32, 48, 64, 100), pick(4, 8, 12, 32, 64, 132),
                          pick(2.0, 5.0, 12.5, 15.0))
        layers.append(bare(layer) if rng.random() < 0.3 else dense(layer, pick(16, 40, 100, 128, 256, 320)))
    return config(int(rng.integers(50, 600)), pick(40, 64, 72, 96, 128, 160, 200), pick(1e-6, 1e-5, 1e-4), pick(1, 2, 3, 4, 6),
                  pick(1, 2, 3, 5, 8), layers)


def draw_tensors(cfg, seed):
    """name -> float32 array (bfloat16 values).  The scales are chosen so that every mechanism matters: attention scores
    have a standard deviation of about 1.8 (a key that is lost or added moves the logits far beyond bfloat16's rounding),
    the streams differ from one another, the heads of an mlstm layer forget at very different speeds, and the taps of the
    convolution are all of one order.

    An mlstm head's read-out is normalised, so where C^T q nearly vanishes (the first token's is (k . q) v: its SIGN is all
    that is left of k . q) rounding decides the result.  Keys are therefore drawn near the queries, which keeps a token's
    product with its own key clear of zero; gates far apart are tested on the mixer alone."""
    rng = np.random.default_rng(seed)
    e, S = cfg["width"], cfg["streams"]
    t = {}

    def mat(out, inp, gain=1.0):
        return rng.normal(0.0, gain / np.sqrt(inp), size=(out, inp))

    def norm(name):
        t[name], t[name + ".b"] = 1.0 + rng.normal(0.0, 0.1, size=e), rng.normal(0.0, 0.2, size=e)

    def streams(name):
        t[name + ".in"] = rng.uniform(0.3, 1.2, size=S) * np.where(rng.random(S) < 0.2, -1.0, 1.0)
        t[name + ".out"] = rng.uniform(0.4, 1.3, size=S)
        t[name + ".mix"] = 0.7 * np.eye(S) + rng.normal(0.0, 0.25, size=(S, S))

    t["embed"] = rng.normal(0.0, 1.0, size=(cfg["vocab"], e))
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        streams(p + "hc1")
        taps = cfg["canon"]["taps"]
        t[p + "canon1"] = rng.normal(0.0, 0.6, size=(e, taps)) / taps ** 0.5
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        x = p + "mix."
        if layer["type"] == "attention":
            G = m["kv_heads"]
            sharp = (1.8 / (m["scale"] * d ** 0.5)) ** 0.5
            t[x + "q"] = mat(H * d, e)
            t[x + "q.norm"] = sharp * (1.0 + rng.normal(0.0, 0.15, size=d))
            t[x + "temp"] = rng.uniform(0.6, 1.5, size=H)
            if m.get("kv_from") is None:
                t[x + "k"], t[x + "v"] = mat(G * d, e), mat(G * dv, e, 1.5)
                t[x + "k.norm"] = sharp * (1.0 + rng.normal(0.0, 0.15, size=d))
        else:
            t[x + "q"] = mat(H * d, e, 1.5)
            t[x + "k"] = t[x + "q"] + mat(H * d, e, 0.7)
            t[x + "v"], t[x + "g"] = mat(H * dv, e, 1.5), mat(H * dv, e, 2.0)
            t[x + "i"], t[x + "f"] = mat(H, e, 0.7), mat(H, e, 0.7)
            t[x + "i.b"] = rng.normal(0.0, 0.7, size=H)
            t[x + "f.b"] = np.array([(7.0, 2.0, 4.0, -1.0)[(h + i) % 4] for h in range(H)])
            t[x + "norm"] = 1.0 + rng.normal(0.0, 0.15, size=H * dv)
        t[x + "o"] = mat(e, H * dv, 2.0)
        f = layer.get("mlp")
        if f:
            norm(p + "norm2")
            streams(p + "hc2")
            t[p + "mlp.gate"], t[p + "mlp.up"] = mat(f["ff"], e, 1.4), mat(f["ff"], e, 1.4)
            t[p + "mlp.down"] = mat(e, f["ff"], 1.4)
    return {n: bf16(a) for n, a in t.items()}


_tmp = []


@functools.lru_cache(maxsize=None)
def model_folder(name):
    """config.json and model.safetensors (bfloat16) of a test configuration, in a temporary place."""
    import torch
    from air_b200.weights.loader import write_model_folder
    d = tempfile.TemporaryDirectory(prefix=f"air_b200_dafotar_{name}_")
    _tmp.append(d)
    if name not in CONFIGS:      # "random<seed>": drawn at random
        seed = int(name[len("random"):])
        CONFIGS[name], SEEDS[name] = random_config(seed), seed
    cfg = CONFIGS[name]
    tensors = {n: torch.from_numpy(np.ascontiguousarray(a)).reshape(a.shape).to(torch.bfloat16)
               for n, a in draw_tensors(cfg, SEEDS[name]).items()}
    write_model_folder(d.name, cfg, tensors)
    return d.name


@functools.lru_cache(maxsize=None)
def plain_model(name):
    from plain import pefivik_plain
    return pefivik_plain.read_model(model_folder(name))


_logits = {}


def plain_logits(name, tokens):
    from plain import dafotar_plain as plain
    key = (name, tuple(tokens))
    if key not in _logits:
        cfg, tensors = plain_model(name)
        _logits[key] = plain.forward(cfg, tensors, list(tokens)).astype(np.float64)
    return _logits[key]


def tokens_for(name, n, seed):
    return np.random.default_rng(9000 + seed).integers(0, CONFIGS[name]["vocab"], size=n).tolist()


def plain_greedy(name, prompt, n):
    out, toks = [], list(prompt)
    for _ in range(n):
        nxt = int(plain_logits(name, toks)[-1].argmax())
        out.append(nxt)
        toks.append(nxt)
    return out


# float32: sums in another order than the 64-bit oracle.  bfloat16: activations rounded to 8 bits at the inputs of the
# products and in the cache, through sharp attention and gates; a request's rows must all be within the row limits, and
# their median within the tighter one.
FP32_TOL = 1e-4
BF16_MAX_TOL = 0.15
BF16_MEAN_TOL = 6e-2
BF16_MEDIAN_TOL = 1e-2


def check(got, name, streams, dtype):
    """got: {(request, position): logits}; every request of `streams` must have rows, and the rows must agree.  Returns the
    largest difference, in units of the largest logit."""
    worst = 0.0
    for rid, toks in streams.items():
        ref = plain_logits(name, toks)
        scale = max(1.0, float(np.abs(ref).max()))
        rows = sorted(p for (r, p) in got if r == rid)
        assert rows, f"no logits for request {rid}"
        means = []
        for p in rows:
            out = got[(rid, p)]
            assert np.isfinite(out).all()
            diff = np.abs(out - ref[p])
            worst = max(worst, float(diff.max()) / scale)
            if dtype == "float32":
                assert diff.max() <= FP32_TOL * scale, (rid, p, float(diff.max()), scale)
            else:
                assert diff.max() <= BF16_MAX_TOL * scale, (rid, p, float(diff.max()), scale)
                assert diff.mean() <= BF16_MEAN_TOL * scale, (rid, p, float(diff.mean()), scale)
                means.append(diff.mean() / scale)
        if len(means) >= 8:
            assert np.median(means) <= BF16_MEDIAN_TOL, (rid, float(np.median(means)))
    return worst
