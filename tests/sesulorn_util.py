"""Set-up of the Sesulorn tests: small configurations that differ in every size and option, model folders with weights
drawn so that a fault shows, and the comparison with the plain implementation."""
import functools
import tempfile

import numpy as np

from bivizen_util import bf16


def attention(heads, kv_heads, dim, vdim, scale, buckets, bias_max):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
                                             bias_max=bias_max, buckets=buckets))


def delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv,
                                                 decay_rank=decay_rank, gate_rank=gate_rank))


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=10000.0):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale)
    if rot_dim:
        m["rot"] = dict(base=base, dims=rot_dim)
    return dict(type="latent_attention", mixer=m)


def dense(layer, ff):
    return dict(layer, mlp=dict(kind="dense", ff=ff))


def bare(layer):
    return dict(layer, mlp=None)


def moe(layer, experts, top, ff, limit, groups=None, shared=None, shared_limit=None):
    f = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    if groups:
        f["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared:
        f["shared"] = dict(ff=shared, limit=shared_limit)
    return dict(layer, mlp=f)


def config(vocab, width, eps, loop, layers):
    d = dict(architecture="Sesulorn", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop:
        d["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return d


# A: the stretch starts at layer 0 and runs three times; values larger than keys and smaller; narrow middles of unequal size
#    that are no multiples of 8; experts in three groups of which two take part; a layer without feed-forward.
# B: no stretch; one head; one tap (no state), narrow middles of one number; a distance table whose last row serves from
#    the sixth position on, and one of two rows; no rotated part; one expert of one, no shared expert; as many key/value
#    heads as heads.
# C: heads of 64 (the dense decoder's tile kernels) with a table that reaches past several tiles, on the model's last
#    layers, which run twice; groups of one expert each; every expert of the kept groups chosen; whole blocks of 128.
# D: no size is a multiple of 4 (the kernels' roads of one element per access); the norm's eps large; a stretch of one pass.
# E: heads of 128 with one key/value head; state heads of more than 128 key channels; a wide latent.
CONFIGS = {
    "A": config(211, 72, 1e-5, (0, 2, 3), [
        moe(attention(6, 2, 16, 20, 0.5, 8, 40), 6, 3, 40, 1.2, groups=(3, 2), shared=48, shared_limit=0.8),
        dense(delta(4, 2, 20, 12, 4, 6, 10), 100),
        bare(latent(3, 24, 8, 20, 40, 28, 0.3, 500.0)),
        moe(delta(2, 2, 12, 16, 3, 5, 9), 8, 3, 24, 2.0, groups=(2, 1)),
        dense(attention(3, 3, 24, 8, 0.4, 6, 30.5), 56)]),
    "B": config(150, 64, 1e-6, None, [
        dense(delta(1, 1, 24, 40, 1, 1, 1), 40),
        moe(attention(1, 1, 32, 24, 0.35, 10, 6), 1, 1, 64, 1.0),
        dense(latent(2, 16, 0, 24, 32, 16, 0.4), 96),
        bare(attention(4, 4, 8, 16, 0.7, 2, 3)),
        moe(latent(1, 8, 16, 40, 24, 40, 0.4, 100.0), 4, 4, 32, 0.7, shared=16, shared_limit=3.0)]),
    "C": config(190, 128, 1e-6, (1, 3, 2), [
        dense(delta(2, 1, 64, 32, 4, 16, 24), 128),
        moe(attention(4, 2, 64, 64, 0.25, 16, 300), 8, 5, 64, 1.5, groups=(8, 5), shared=128, shared_limit=1.5),
        dense(latent(4, 32, 16, 48, 64, 96, 0.3), 256)]),
    "D": config(133, 90, 1e-3, (1, 3, 1), [
        dense(attention(3, 1, 14, 10, 0.5, 14, 60), 50),
        moe(latent(3, 10, 6, 14, 22, 18, 0.4, 1000.0), 6, 2, 30, 1.1, groups=(2, 2), shared=22, shared_limit=2.2),
        dense(delta(3, 1, 10, 6, 6, 3, 7), 34)]),
    "E": config(300, 256, 1e-6, (0, 1, 2), [
        dense(attention(4, 1, 128, 128, 0.17, 32, 128), 320),
        dense(delta(2, 2, 136, 72, 2, 32, 40), 256),
        bare(latent(8, 32, 32, 32, 128, 64, 0.25, 50000.0))]),
}
SEEDS = {"A": 61, "B": 62, "C": 63, "D": 64, "E": 65}


def random_config(seed):
    """A configuration drawn at random: 2 to 6 layers in any order, a repeated stretch anywhere (or none), every size and
    constant from a list that includes 1, equal and unequal sizes and sizes that are no multiples of 8 or 16."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers = []
    for i in range(int(rng.integers(2, 7))):
        kind = int(rng.integers(3))
        if kind == 0:
            dim, kv = pick(8, 16, 24, 32, 64, 128), pick(1, 2, 3)
            rows = pick(2, 4, 8, 10, 32)
            layer = attention(kv * pick(1, 2, 3, 4), kv, dim, pick(8, 16, 24, 40, 64, dim, dim), pick(1.5, 2.0, 2.5) / dim ** 0.5,
                              rows, rows // 2 + pick(1, 5, 20, 100, 400))
        elif kind == 1:
            kv = pick(1, 2, 3)
            layer = delta(kv * pick(1, 2), kv, pick(4, 8, 20, 32, 48, 64, 100), pick(4, 8, 12, 32, 64, 132), pick(1, 2, 3, 4, 7),
                          pick(1, 4, 6, 16, 24), pick(1, 3, 8, 20))
        else:
            layer = latent(pick(1, 2, 3, 4, 8), pick(8, 16, 24, 32, 64), pick(0, 2, 8, 16, 32), pick(8, 16, 24, 40, 64),
                           pick(8, 24, 40, 56, 96, 128), pick(8, 12, 24, 64, 100), pick(0.25, 0.35), pick(100.0, 10000.0, 500000.0))
        u = rng.random()
        if u < 0.15:
            layers.append(bare(layer))
        elif u < 0.5:
            layers.append(dense(layer, pick(16, 40, 100, 128, 256, 320)))
        else:
            count, size = pick(1, 2, 3, 4), pick(1, 2, 3, 4)
            keep = int(rng.integers(1, count + 1))
            layers.append(moe(layer, count * size, int(rng.integers(1, keep * size + 1)), pick(16, 24, 40, 64, 100),
                              pick(0.5, 1.0, 1.7, 7.0), groups=(count, keep) if count > 1 or rng.random() < 0.5 else None,
                              shared=None if rng.random() < 0.3 else pick(16, 40, 64, 96, 128), shared_limit=pick(0.6, 1.3, 4.0)))
    n = len(layers)
    loop = None
    if rng.random() < 0.8:
        start = int(rng.integers(0, n))
        loop = (start, int(rng.integers(start + 1, n + 1)), pick(1, 2, 2, 3))
    return config(int(rng.integers(50, 700)), pick(40, 64, 72, 96, 128, 160, 200), pick(1e-6, 1e-5, 1e-4), loop, layers)


ROUTE_CHANNELS = (1.0, 0.52, 0.27, 0.14, 0.075)


def _bits(n):
    return max(0, int(np.ceil(np.log2(n)))) if n > 1 else 0


def mixer_tensors(rng, e, layer, keep=()):
    """name behind 'mix.' -> array: scales chosen so that every mechanism matters.  keep: rows of the output matrix that are
    zero (columns of the stream that the layer leaves alone).

    A state head's read-out is normalised, so where S^T q nearly vanishes (the first token's is (k . q) v) rounding decides
    the result: keys are drawn near the queries, their convolutions too."""
    m = layer["mixer"]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    mat = lambda out, inp, gain=1.0: rng.normal(0.0, gain / np.sqrt(inp), size=(out, inp))
    t = {}
    if layer["type"] == "attention":
        G = m["kv_heads"]
        t["q"], t["k"], t["v"] = mat(H * d, e), mat(G * d, e), mat(G * dv, e, 1.5)
        t["q.b"], t["k.b"], t["v.b"] = (rng.normal(0.0, 0.5, size=n) for n in (H * d, G * d, G * dv))
        t["rel"] = rng.normal(0.0, 1.5, size=(m["buckets"], H))
    elif layer["type"] == "channel_delta":
        G, ra, rg = m["kv_heads"], m["decay_rank"], m["gate_rank"]
        t["q"] = mat(G * d, e, 1.5)
        t["k"] = t["q"] + mat(G * d, e, 0.6)
        t["v"] = mat(H * dv, e, 1.5)
        taps = m["conv"]
        t["q.conv"] = rng.normal(0.0, 0.6, size=(G * d, taps)) / taps ** 0.5
        t["q.conv"][:, -1] += 1.0
        t["k.conv"] = t["q.conv"] + rng.normal(0.0, 0.2, size=(G * d, taps)) / taps ** 0.5
        t["v.conv"] = rng.normal(0.0, 1.0, size=(H * dv, taps)) / taps ** 0.5
        t["b"] = mat(H, e, 1.5)
        t["A_log"] = rng.uniform(-1.5, 0.7, size=H)
        # channels that forget at very different speeds: some hardly in hundreds of tokens, some at once
        t["dt_bias"] = rng.choice([-7.0, -4.0, -1.0, 1.5], size=H * d) + rng.normal(0.0, 0.3, size=H * d)
        t["a1"], t["a2"] = mat(ra, e), mat(H * d, ra, 1.2)
        t["g1"], t["g2"] = mat(rg, e), mat(H * dv, rg, 2.0)
        t["norm"] = 1.0 + rng.normal(0.0, 0.15, size=dv)
    else:
        R, Q, r = m["kv_rank"], m["q_rank"], m["rot_dim"]
        sharp = (2.0 / (m["scale"] * (d + r) ** 0.5)) ** 0.5
        t["dq"], t["dq.norm"] = mat(Q, e, 2.0), 1.0 + rng.normal(0.0, 0.15, size=Q)
        t["uq"] = mat(H * (d + r), Q, sharp)
        t["dkv"], t["dkv.norm"] = mat(R + r, e, 1.0), 1.0 + rng.normal(0.0, 0.15, size=R)
        t["dkv"][R:] *= sharp
        t["uk"], t["uv"] = mat(H * d, R, sharp), mat(H * dv, R, 1.5)
    t["o"] = mat(e, H * dv, 1.2)
    t["o"][list(keep)] = 0.0
    return t


def draw_tensors(cfg, seed):
    """name -> float32 array (bfloat16 values).

    A router is a discontinuity: with random router weights one token in a hundred has two experts so close that
    bfloat16's rounding picks the other one, and the logits then differ by a whole expert.  So the routers here decide by
    a few channels of the stream that only the token table touches (output matrices leave them alone, loop.in hands them on):
    a token carries a sign pattern with falling magnitudes there, and an expert's router row the pattern of its index, the
    bits of its place in the group on the channels with the large magnitudes and the bits of its group behind them.  A
    last channel is zero in the stream and has the negative sum of a row's pattern, which takes the row's mean out of the
    choice.  Every group holds the same places, so the order of the groups' best experts is the order of their own bits,
    while without groups the experts at the best place of every group would be taken.
    Which experts a token takes is then a matter of the token, clear of rounding; their scores still depend on everything,
    through the norm and the rest of the router row."""
    rng = np.random.default_rng(seed)
    e = cfg["width"]
    t = {}
    bits = 0
    for layer in cfg["layers"]:
        f = layer.get("mlp")
        if f and f["kind"] == "moe":
            g = (f["router"].get("groups") or {"count": 1})["count"]
            bits = max(bits, _bits(g) + _bits(f["router"]["experts"] // g))
    assert bits <= len(ROUTE_CHANNELS)
    nr = bits + 1 if bits else 0
    keep = list(range(nr))

    def mat(out, inp, gain=1.0):
        return rng.normal(0.0, gain / np.sqrt(inp), size=(out, inp))

    def norm(name):
        w, b = 1.0 + rng.normal(0.0, 0.1, size=e), rng.normal(0.0, 0.2, size=e)
        w[:nr], b[:nr] = 1.0, 0.0
        t[name], t[name + ".b"] = w, b

    t["embed"] = rng.normal(0.0, 1.0, size=(cfg["vocab"], e))
    tokens = np.arange(cfg["vocab"])
    for c in range(bits):
        t["embed"][:, c] = np.where((tokens >> c) & 1, 1.0, -1.0) * ROUTE_CHANNELS[c] * 1.5
    t["embed"][:, bits:nr] = 0.0
    if cfg.get("loop"):
        t["loop.in"] = mat(e, 2 * e, 1.0) + 0.6 * np.concatenate([np.eye(e), np.eye(e)], axis=1)
        t["loop.in"][:nr] = 0.0
        for c in keep:
            t["loop.in"][c, e + c] = 1.0
    t["head"] = mat(cfg["vocab"], e, 2.0)
    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        norm(p + "norm1")
        t.update({p + "mix." + n: a for n, a in mixer_tensors(rng, e, layer, keep).items()})
        f = layer.get("mlp")
        if not f:
            continue
        if f["kind"] == "dense":
            t[p + "mlp.gate"], t[p + "mlp.up"] = mat(f["ff"], e, 1.4), mat(f["ff"], e, 1.4)
            t[p + "mlp.down"] = mat(e, f["ff"], 1.2)
            t[p + "mlp.down"][:nr] = 0.0
            continue
        r = f["router"]
        n = r["experts"]
        g = (r.get("groups") or {"count": 1})["count"]
        size, gb = n // g, _bits(g)
        t[p + "mlp.router"] = mat(n, e, 0.02)
        for x in range(n):
            code = [(x % size >> c) & 1 for c in range(_bits(size))] + [(x // size >> c) & 1 for c in range(gb)]
            code = [(1.0 if b else -1.0) * 1.5 for b in code]
            if nr:
                t[p + "mlp.router"][x, :nr] = 0.0
                t[p + "mlp.router"][x, :len(code)] = code
                t[p + "mlp.router"][x, bits] = -sum(code)
            q = f"{p}mlp.e{x}."
            t[q + "gate"], t[q + "up"] = mat(f["expert"]["ff"], e, 1.5), mat(f["expert"]["ff"], e, 1.5)
            t[q + "down"] = mat(e, f["expert"]["ff"], 1.5)
            t[q + "down"][:nr] = 0.0
        if f.get("shared"):
            s, q = f["shared"]["ff"], p + "mlp.shared."
            t[q + "gate"], t[q + "up"], t[q + "sg"] = mat(s, e, 1.5), mat(s, e, 1.5), mat(1, e, 1.5)
            t[q + "down"] = mat(e, s, 1.0)
            t[q + "down"][:nr] = 0.0
    return {n: bf16(a) for n, a in t.items()}


_tmp = []


@functools.lru_cache(maxsize=None)
def model_folder(name):
    """config.json and model.safetensors (bfloat16) of a test configuration, in a temporary place.  config.json is written
    without the sizes that are only the shapes of tensors."""
    import torch
    from air_b200.weights.loader import write_model_folder
    d = tempfile.TemporaryDirectory(prefix=f"air_b200_sesulorn_{name}_")
    _tmp.append(d)
    if name not in CONFIGS:      # "random<seed>": drawn at random
        seed = int(name[len("random"):])
        CONFIGS[name], SEEDS[name] = random_config(seed), seed
    cfg = CONFIGS[name]
    tensors = {n: torch.from_numpy(np.ascontiguousarray(a)).reshape(a.shape).to(torch.bfloat16)
               for n, a in draw_tensors(cfg, SEEDS[name]).items()}
    bare_layers = [dict(l, mixer={k: v for k, v in l["mixer"].items() if k not in ("buckets", "decay_rank", "gate_rank")})
                   for l in cfg["layers"]]
    write_model_folder(d.name, dict(cfg, layers=bare_layers), tensors)
    return d.name


@functools.lru_cache(maxsize=None)
def plain_model(name):
    from plain import pefivik_plain
    return pefivik_plain.read_model(model_folder(name))


_logits = {}


def plain_logits(name, tokens):
    from plain import sesulorn_plain as plain
    key = (name, tuple(tokens))
    if key not in _logits:
        cfg, tensors = plain_model(name)
        _logits[key] = plain.forward(cfg, tensors, list(tokens)).astype(np.float64)
    return _logits[key]


def tokens_for(name, n, seed):
    return np.random.default_rng(9100 + seed).integers(0, CONFIGS[name]["vocab"], size=n).tolist()


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
FP32_TOL = 2e-5
BF16_MAX_TOL = 0.1
BF16_MEAN_TOL = 3e-2
BF16_MEDIAN_TOL = 8e-3


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
