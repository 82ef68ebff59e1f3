"""Mixers that keep a state of fixed size per request instead of keys and values: a matrix per head that every
token updates and reads (linear attention with gates), and the short convolutions in front of it."""
from __future__ import annotations

import numpy as np
import torch

from ..config.model_config import ConfigError
from ..csrc import ops
from ..weights.loader import TensorSpec
from .base import HostBatch, Mixer, Plan, SlotState
from .linear import Linear
from .registry import register_mixer


class _StateMixer(Mixer):
    """What the two mixers below share: one product for all their projections of the layer's input, a 32-bit state
    [heads, head_dim, v_dim] per request, and the norm with a gate that follows the read-out."""

    graph_safe = True

    def _project(self, tensors, names, rt):
        ws = [tensors[self.prefix + n] for n in names]
        if len({w.dtype for w in ws}) != 1:
            raise ValueError(f"{self.prefix}: the projections are stored in different precisions")
        self.proj = Linear(torch.cat(ws, dim=0).contiguous(), rt.status)
        self.columns, at = {}, 0
        for n, w in zip(names, ws):
            self.columns[n] = (at, at + w.shape[0])
            at += w.shape[0]

    def _band(self, proj, name):
        lo, hi = self.columns[name]
        return proj[:, lo:hi]

    def _finish(self, o, gate, ctx, sigmoid=False):
        """norm over each head's read-out, times the weight and silu(gate) (or sigmoid(gate)), then the output projection"""
        T = o.shape[0]
        y = torch.empty((T, self.heads * self.v_dim), dtype=self.rt.dtype, device=o.device)
        ops.gated_rmsnorm(o, gate, self.norm_weight, self.eps, y, ctx.token_seq, sigmoid=sigmoid)
        return self.o.f32_sums(y)

    def _convolved(self, proj, tail, ctx):
        """The first `channels` columns of proj behind the short convolution and SiLU; tail: the state of its last inputs."""
        y = torch.empty((proj.shape[0], self.channels), dtype=torch.float32, device=proj.device)
        state = tail.state if self.taps > 1 else tail.state[:, :, :0].contiguous()
        return ops.short_conv_silu(proj[:, :self.channels], self.conv_weight, state, y, ctx.q_start, ctx.slots, ctx.max_q_len)


@register_mixer("gated_delta")
class GatedDeltaRule(_StateMixer):
    """The gated delta rule.  q, k (kv_heads x head_dim) and v (heads x v_dim) are projections of the input followed by
    a short causal convolution over time per channel (`conv` taps, the last one the current token's) and SiLU; q and k
    are scaled to unit length per head (x / sqrt(sum x^2 + 1e-6)), q also by head_dim^-1/2; head h reads q/k head
    h // (heads / kv_heads).  Per head and token, with b = sigmoid(W_b x) and
    g = exp(-exp(A_log) * softplus(W_a x + dt_bias)):

        S = g S;   u = b (v - S^T k);   S = S + k u^T;   o = S^T q

    then o / sqrt(mean(o^2) + eps) * norm * silu(W_g x), and the output projection.  S and the convolutions' last
    conv - 1 inputs are the request's state, 32-bit, zero at its start.

    params: hidden, heads, kv_heads, head_dim, v_dim, conv, eps.  Tensors: <prefix>q, k, v, each with <name>.conv
    [channels, conv]; b, a [heads, hidden]; A_log, dt_bias [heads]; norm [v_dim]; g [heads*v_dim, hidden];
    o [hidden, heads*v_dim]."""

    def __init__(self, spec, prefix=""):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden, self.heads, self.kv_heads = p["hidden"], p["heads"], p["kv_heads"]
        self.head_dim, self.v_dim, self.taps, self.eps = p["head_dim"], p["v_dim"], int(p["conv"]), float(p["eps"])
        if self.heads % self.kv_heads:
            raise ConfigError("data_error", "gated_delta: heads must be a multiple of kv_heads")
        if not (1 <= self.taps <= 16):
            raise ConfigError("unsupported", f"gated_delta: a convolution of {self.taps} taps (the kernel takes 1 to 16)")
        if self.head_dim > 1024:
            raise ConfigError("unsupported", f"gated_delta: {self.head_dim} key channels per head (up to 1,024)")
        self.channels = 2 * self.kv_heads * self.head_dim + self.heads * self.v_dim

    def cache_needs(self):
        return (SlotState((self.heads, self.head_dim, self.v_dim)),
                SlotState((self.channels, max(self.taps - 1, 1))))

    def tensor_specs(self):
        p, e, H, G, d, dv = self.prefix, self.hidden, self.heads, self.kv_heads, self.head_dim, self.v_dim
        rows = {"q": G * d, "k": G * d, "v": H * dv}
        specs = []
        for n in "qkv":
            specs += [TensorSpec(p + n, (rows[n], e)), TensorSpec(p + n + ".conv", (rows[n], self.taps), wide=True, std=0.3)]
        specs += [TensorSpec(p + "b", (H, e)), TensorSpec(p + "A_log", (H,), wide=True),
                  TensorSpec(p + "norm", (dv,), init="one_plus_normal", wide=True), TensorSpec(p + "a", (H, e)),
                  TensorSpec(p + "dt_bias", (H,), wide=True), TensorSpec(p + "g", (H * dv, e)),
                  TensorSpec(p + "o", (e, H * dv))]
        return specs

    def load(self, tensors, rt):
        super().load(tensors, rt)
        p = self.prefix
        self._project(tensors, ["q", "k", "v", "b", "a", "g"], rt)
        f32 = lambda n: tensors[p + n].to(torch.float32).contiguous()
        self.conv_weight = torch.cat([f32(n + ".conv") for n in "qkv"], dim=0).contiguous()
        self.a_log, self.dt_bias, self.norm_weight = f32("A_log"), f32("dt_bias"), f32("norm")
        self.o = Linear(tensors[p + "o"], rt.status)

    def forward(self, x, ctx, cache, owns_cache=True):
        state, tail = cache
        T, H, G, d, dv = x.shape[0], self.heads, self.kv_heads, self.head_dim, self.v_dim
        proj = self.proj.f32(x)
        y = self._convolved(proj, tail, ctx)
        o = torch.empty((T, H, dv), dtype=torch.float32, device=x.device)
        ops.linear_scan(ops.SCAN_DELTA, y[:, :G * d], y[:, G * d:2 * G * d], y[:, 2 * G * d:],
                        self._band(proj, "a"), state.state, o, ctx.q_start, ctx.slots, ctx.token_seq, q_scale=d ** -0.5,
                        beta=self._band(proj, "b"), a_log=self.a_log, dt_bias=self.dt_bias, unit=True, unit_eps=1e-6)
        return self._finish(o, self._band(proj, "g"), ctx)


@register_mixer("channel_delta")
class ChannelDeltaRule(_StateMixer):
    """The delta rule with a decay per key channel.  q, k, v, their convolutions, unit lengths and b as in GatedDeltaRule; the
    decay of channel c of head h is g = exp(-exp(A_log_h) * softplus(W_a2 (W_a1 x) + dt_bias)), a product through a narrow
    middle laid out heads x head_dim, and scales row c of the head's state:

        S = diag(g) S;   u = b (v - S^T k);   S = S + k u^T;   o = S^T q

    then o / sqrt(mean(o^2) + eps) * norm, times sigmoid(W_g2 (W_g1 x)) (laid out heads x v_dim), and the output
    projection.  S and the convolutions' last conv - 1 inputs are the request's state, 32-bit, zero at its start.

    In a bfloat16 engine portions of PORTION tokens or more are taken in chunks whose rows are computed side by side
    (ops.delta_portions); everything else goes token by token (ops.linear_scan).

    The two products out of a narrow middle take its numbers as they left the first product: a float32 engine in 32-bit,
    a bfloat16 engine as two bfloat16 halves side by side, against the matrix twice (ops.split_bands), so that the
    decays are 32-bit but for the weights' own precision.

    params: hidden, heads, kv_heads, head_dim, v_dim, conv, decay_rank, gate_rank (the narrow middles), eps.  Tensors:
    <prefix>q, k, v, each with <name>.conv [channels, conv]; b [heads, hidden]; A_log [heads]; dt_bias [heads*head_dim];
    a1 [decay_rank, hidden]; a2 [heads*head_dim, decay_rank]; g1 [gate_rank, hidden]; g2 [heads*v_dim, gate_rank]; norm
    [v_dim]; o [hidden, heads*v_dim]."""

    def __init__(self, spec, prefix=""):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden, self.heads, self.kv_heads = p["hidden"], p["heads"], p["kv_heads"]
        self.head_dim, self.v_dim, self.taps, self.eps = p["head_dim"], p["v_dim"], int(p["conv"]), float(p["eps"])
        self.decay_rank, self.gate_rank = int(p["decay_rank"]), int(p["gate_rank"])
        if self.heads % self.kv_heads:
            raise ConfigError("data_error", "channel_delta: heads must be a multiple of kv_heads")
        if not (1 <= self.taps <= 16):
            raise ConfigError("unsupported", f"channel_delta: a convolution of {self.taps} taps (the kernel takes 1 to 16)")
        if self.head_dim > 1024:
            raise ConfigError("unsupported", f"channel_delta: {self.head_dim} key channels per head (up to 1,024)")
        self.channels = 2 * self.kv_heads * self.head_dim + self.heads * self.v_dim

    def cache_needs(self):
        return (SlotState((self.heads, self.head_dim, self.v_dim)),
                SlotState((self.channels, max(self.taps - 1, 1))))

    def tensor_specs(self):
        p, e, H, G, d, dv = self.prefix, self.hidden, self.heads, self.kv_heads, self.head_dim, self.v_dim
        rows = {"q": G * d, "k": G * d, "v": H * dv}
        specs = []
        for n in "qkv":
            specs += [TensorSpec(p + n, (rows[n], e)), TensorSpec(p + n + ".conv", (rows[n], self.taps), wide=True, std=0.3)]
        return specs + [
            TensorSpec(p + "b", (H, e)), TensorSpec(p + "A_log", (H,), wide=True), TensorSpec(p + "dt_bias", (H * d,), wide=True),
            TensorSpec(p + "a1", (self.decay_rank, e)), TensorSpec(p + "a2", (H * d, self.decay_rank), std=0.3),
            TensorSpec(p + "g1", (self.gate_rank, e)), TensorSpec(p + "g2", (H * dv, self.gate_rank), std=0.3),
            TensorSpec(p + "norm", (dv,), init="one_plus_normal", wide=True), TensorSpec(p + "o", (e, H * dv))]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        p, w = self.prefix, tensors[self.prefix + "q"]
        # rows of zeros: the narrow middles are filled up to multiples of 4 numbers (the second products' inner size, two
        # halves each, is then one of 8), the matrix up to a multiple of 8 rows, which the tensor-core kernels want
        tensors = dict(tensors)

        def zeros(name, rows):
            if rows:
                tensors[p + name] = torch.zeros((rows, self.hidden), dtype=w.dtype, device=w.device)
            return [name] * (rows > 0)

        self.middle = tuple(r + (-r % 4) for r in (self.decay_rank, self.gate_rank))
        bands = ["q", "k", "v", "b"]
        bands += zeros("pad.b", -sum(tensors[p + n].shape[0] for n in bands) % 4)
        bands += ["a1"] + zeros("pad.a", self.middle[0] - self.decay_rank)
        bands += ["g1"] + zeros("pad.g", self.middle[1] - self.gate_rank)
        bands += zeros("pad", -sum(tensors[p + n].shape[0] for n in bands) % 8)
        self._project(tensors, bands, rt)
        f32 = lambda n: tensors[p + n].to(torch.float32).contiguous()
        self.conv_weight = torch.cat([f32(n + ".conv") for n in "qkv"], dim=0).contiguous()
        self.a_log, self.dt_bias, self.norm_weight = f32("A_log"), f32("dt_bias"), f32("norm")
        self.a2, self.g2 = (self._out_of_the_middle(tensors[p + n], r, rt) for n, r in zip(("a2", "g2"), self.middle))
        self.o = Linear(tensors[p + "o"], rt.status)

    @staticmethod
    def _out_of_the_middle(m, width, rt):
        """The second product as a Linear: its inner size filled up with zeros, and in a bfloat16 engine the matrix twice; its
        rows filled up to a multiple of 4."""
        rows, rank = m.shape
        twice = 1 if m.dtype == torch.float32 else 2
        full = torch.zeros((rows + (-rows % 4), twice * width), dtype=m.dtype, device=m.device)
        for i in range(twice):
            full[:rows, i * width:i * width + rank] = m
        return Linear(full, rt.status)

    PORTION = 24

    def plan_key(self):
        chunks = self.rt.dtype == torch.bfloat16 and self.head_dim <= ops.DELTA_MAX_D
        return ("channel_delta.chunks", self.PORTION) if chunks else None

    def plan(self, batch: HostBatch) -> Plan:
        """portions [L, 4] = (first row, tokens, slot, first chunk) of the entries of at least PORTION tokens, chunks [N, 2] =
        (first row, tokens) of theirs; short_slots: the slot of every other entry, short_seq: of their rows, -1 elsewhere."""
        portions, chunks, short_slots = [], [], []
        short_seq = np.full(batch.q_start[-1], -1, dtype=np.int32)
        for i, n in enumerate(batch.counts):
            first = batch.q_start[i]
            if n < self.PORTION:
                short_slots.append(batch.slots[i])
                short_seq[first:first + n] = batch.slots[i]
                continue
            short_slots.append(-1)
            portions.append((first, n, batch.slots[i], len(chunks)))
            chunks += [(first + at, min(ops.DELTA_CHUNK, n - at)) for at in range(0, n, ops.DELTA_CHUNK)]
        return Plan(arrays={"portions": np.asarray(portions, dtype=np.int32).reshape(-1, 4),
                            "chunks": np.asarray(chunks, dtype=np.int32).reshape(-1, 2),
                            "short_slots": np.asarray(short_slots, dtype=np.int32), "short_seq": short_seq},
                    values={"long": bool(portions), "short": len(portions) < len(batch.counts)})

    def _narrow(self, proj):
        """(decay logits [T, heads*head_dim], gate logits [T, heads*v_dim]), float32."""
        at, (ra, rg) = self.columns["a1"][0], self.middle
        if self.a2.weight.dtype == torch.float32:
            za, zg = (lin(proj[:, lo:lo + r].contiguous(), torch.float32)
                      for lin, lo, r in ((self.a2, at, ra), (self.g2, at + ra, rg)))
        else:
            a, g = ops.split_bands(proj[:, at:at + ra + rg], ra, rg)
            za, zg = self.a2.f32(a), self.g2.f32(g)
        return za[:, :self.heads * self.head_dim], zg[:, :self.heads * self.v_dim]

    def forward(self, x, ctx, cache, owns_cache=True):
        state, tail = cache
        T, H, G, d, dv = x.shape[0], self.heads, self.kv_heads, self.head_dim, self.v_dim
        proj = self.proj.f32(x)
        y = self._convolved(proj, tail, ctx)
        decay, gate = self._narrow(proj)
        o = torch.empty((T, H, dv), dtype=torch.float32, device=x.device)
        bands = (y[:, :G * d], y[:, G * d:2 * G * d], y[:, 2 * G * d:], decay, state.state, o)
        numbers = dict(q_scale=d ** -0.5, beta=self._band(proj, "b"), a_log=self.a_log, dt_bias=self.dt_bias, unit_eps=1e-6)
        plan = ctx.plans.get(self.plan_key()) if self.plan_key() is not None else None
        if plan is None or not plan.long:
            ops.linear_scan(ops.SCAN_CHANNEL_DELTA, *bands, ctx.q_start, ctx.slots, ctx.token_seq, unit=True, **numbers)
        else:
            if plan.short:
                ops.linear_scan(ops.SCAN_CHANNEL_DELTA, *bands, ctx.q_start, plan.short_slots, plan.short_seq, unit=True,
                                **numbers)
            ops.delta_portions(*bands, plan.portions, plan.chunks, status=ctx.status, **numbers)
        return self._finish(o, gate, ctx, sigmoid=True)


@register_mixer("gla")
class GatedLinearAttention(_StateMixer):
    """Gated linear attention.  q = W_q x * head_dim^-1/2, k = W_k x (heads x head_dim), v = W_v x (heads x v_dim);
    a decay per key channel, alpha = sigmoid(W_a2 (W_a1 x) + b_a2)^(1/tau) (a product through a narrow middle);
    per head and token

        S = diag(alpha) S + k v^T;   o = S^T q

    then o / sqrt(mean(o^2) + eps) * norm, times silu(W_g x), and the output projection.  S is the request's state,
    32-bit, zero at its start.  The decay's second product, its sigmoid, logarithm and power are 32-bit.

    params: hidden, heads, head_dim, v_dim, tau, rank (the narrow middle), eps.  Tensors: <prefix>q, k
    [heads*head_dim, hidden]; v, g [heads*v_dim, hidden]; a1 [rank, hidden]; a2 [heads*head_dim, rank]; a2.b
    [heads*head_dim]; norm [v_dim]; o [hidden, heads*v_dim]."""

    def __init__(self, spec, prefix=""):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden, self.heads, self.head_dim, self.v_dim = p["hidden"], p["heads"], p["head_dim"], p["v_dim"]
        self.tau, self.rank, self.eps = float(p["tau"]), int(p["rank"]), float(p["eps"])
        if self.head_dim > 1024:
            raise ConfigError("unsupported", f"gla: {self.head_dim} key channels per head (up to 1,024)")
        if not (self.tau > 0.0):
            raise ConfigError("data_error", "gla: tau must be positive")

    def cache_needs(self):
        return (SlotState((self.heads, self.head_dim, self.v_dim)),)

    def tensor_specs(self):
        p, e, H, d, dv, r = self.prefix, self.hidden, self.heads, self.head_dim, self.v_dim, self.rank
        return [TensorSpec(p + "q", (H * d, e)), TensorSpec(p + "k", (H * d, e)), TensorSpec(p + "v", (H * dv, e)),
                TensorSpec(p + "g", (H * dv, e)), TensorSpec(p + "o", (e, H * dv)),
                TensorSpec(p + "norm", (dv,), init="one_plus_normal", wide=True), TensorSpec(p + "a1", (r, e)),
                TensorSpec(p + "a2", (H * d, r), wide=True, std=0.3), TensorSpec(p + "a2.b", (H * d,), wide=True)]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        p = self.prefix
        self._project(tensors, ["q", "k", "v", "g", "a1"], rt)
        f32 = lambda n: tensors[p + n].to(torch.float32).contiguous()
        self.a2, self.a2_bias, self.norm_weight = f32("a2"), f32("a2.b"), f32("norm")
        self.o = Linear(tensors[p + "o"], rt.status)

    def forward(self, x, ctx, cache, owns_cache=True):
        (state,) = cache
        T, H, d, dv = x.shape[0], self.heads, self.head_dim, self.v_dim
        proj = self.proj.f32(x)
        z = torch.empty((T, H * d), dtype=torch.float32, device=x.device)
        ops.gemm_f32(self._band(proj, "a1").contiguous(), self.a2, self.a2_bias, z)
        o = torch.empty((T, H, dv), dtype=torch.float32, device=x.device)
        ops.linear_scan(ops.SCAN_GLA, self._band(proj, "q"), self._band(proj, "k"), self._band(proj, "v"), z,
                        state.state, o, ctx.q_start, ctx.slots, ctx.token_seq, q_scale=d ** -0.5, tau=self.tau)
        return self._finish(o, self._band(proj, "g"), ctx)


@register_mixer("hgrn2")
class HGRN2(_StateMixer):
    """HGRN2: gated linear attention without a key projection; what a channel does not keep of its old state (1 - f) is
    the share of the new value that it takes in.  q = silu(W_q x) (heads x
    head_dim), v = W_v x (heads x v_dim); per head and channel f = l + (1 - l) sigmoid(W_f x + b_f) with a learned lower
    bound l; per head and token

        S = diag(f) S + (1 - f) v^T;   o = S^T q

    (k is not a projection and q carries no factor), then o / sqrt(mean(o^2) + eps) * norm over each head's v_dim numbers (one weight for all
    heads, no gate) and the output projection.  S is the request's state, 32-bit, zero at its start.  The gate, its
    sigmoid and 1 - f are 32-bit; the recurrence is gated linear attention's with k = 1 - f.

    params: hidden, heads, head_dim, v_dim, eps.  Tensors: <prefix>q, f [heads*head_dim, hidden]; f.b, lower
    [heads*head_dim]; v [heads*v_dim, hidden]; norm [v_dim]; o [hidden, heads*v_dim]."""

    def __init__(self, spec, prefix=""):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden, self.heads, self.head_dim, self.v_dim = p["hidden"], p["heads"], p["head_dim"], p["v_dim"]
        self.eps = float(p["eps"])
        if self.head_dim > 1024:
            raise ConfigError("unsupported", f"hgrn2: {self.head_dim} channels per head (up to 1,024)")

    def cache_needs(self):
        return (SlotState((self.heads, self.head_dim, self.v_dim)),)

    def tensor_specs(self):
        p, e, H, d, dv = self.prefix, self.hidden, self.heads, self.head_dim, self.v_dim
        return [TensorSpec(p + "q", (H * d, e)), TensorSpec(p + "f", (H * d, e)), TensorSpec(p + "f.b", (H * d,), wide=True),
                TensorSpec(p + "lower", (H * d,), init="uniform", std=0.9, wide=True), TensorSpec(p + "v", (H * dv, e)),
                TensorSpec(p + "norm", (dv,), init="one_plus_normal", wide=True), TensorSpec(p + "o", (e, H * dv))]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        p = self.prefix
        self._project(tensors, ["q", "f", "v"], rt)
        f32 = lambda n: tensors[p + n].to(torch.float32).contiguous()
        self.gate_bias, self.lower, self.norm_weight = f32("f.b"), f32("lower"), f32("norm")
        self.o = Linear(tensors[p + "o"], rt.status)

    def forward(self, x, ctx, cache, owns_cache=True):
        (state,) = cache
        T, H, dv = x.shape[0], self.heads, self.v_dim
        proj = self.proj.f32(x)
        o = torch.empty((T, H, dv), dtype=torch.float32, device=x.device)
        ops.linear_scan(ops.SCAN_HGRN, self._band(proj, "q"), None, self._band(proj, "v"), self._band(proj, "f"),
                        state.state, o, ctx.q_start, ctx.slots, ctx.token_seq, lower=self.lower,
                        gate_bias=self.gate_bias)
        y = torch.empty((T, H * dv), dtype=self.rt.dtype, device=o.device)
        ops.gated_rmsnorm(o, None, self.norm_weight, self.eps, y, ctx.token_seq)
        return self.o.f32_sums(y)


@register_mixer("retention")
class Retention(_StateMixer):
    """Retention: linear attention with one constant decay per head and neither softmax nor denominator.  q = W_q x,
    k = W_k x (heads x head_dim), v = W_v x (heads x v_dim); q and k are rotated by the token's position (the position
    encoding's frequencies, the first part of a head), k is then multiplied by head_dim^-1/2; per head and token

        S = g_h S + k v^T;   o = S^T q

    with g_h the head's entry of `decay`; then each head's o over its root mean square (o / sqrt(mean(o^2) + eps), no
    weight), times silu(W_g x), and the output projection.  S is the request's state, 32-bit, zero at its start.  The
    rotation, the state and the norm are 32-bit.

    params: hidden, heads, head_dim, v_dim, decay (a number per head), eps, position (a position encoding that gives
    64-bit frequencies, or none).  Tensors: <prefix>q, k [heads*head_dim, hidden]; v, g [heads*v_dim, hidden];
    o [hidden, heads*v_dim]."""

    def __init__(self, spec, prefix=""):
        super().__init__(spec, prefix)
        from .registry import POSITION_ENCODINGS
        p = spec.params
        self.hidden, self.heads, self.head_dim, self.v_dim = p["hidden"], p["heads"], p["head_dim"], p["v_dim"]
        self.eps = float(p["eps"])
        self.decay = tuple(float(g) for g in p["decay"])
        if len(self.decay) != self.heads:
            raise ConfigError("data_error", f"retention: {len(self.decay)} decays for {self.heads} heads")
        if self.head_dim > 1024:
            raise ConfigError("unsupported", f"retention: {self.head_dim} key channels per head (up to 1,024)")
        pos = p.get("position")
        self.position = POSITION_ENCODINGS.get(pos.kind)(pos) if pos is not None else None

    def cache_needs(self):
        return (SlotState((self.heads, self.head_dim, self.v_dim)),)

    def tensor_specs(self):
        p, e, H, d, dv = self.prefix, self.hidden, self.heads, self.head_dim, self.v_dim
        return [TensorSpec(p + "q", (H * d, e)), TensorSpec(p + "k", (H * d, e)), TensorSpec(p + "v", (H * dv, e)),
                TensorSpec(p + "g", (H * dv, e)), TensorSpec(p + "o", (e, H * dv))]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        self._project(tensors, ["q", "k", "v", "g"], rt)
        self.o = Linear(tensors[self.prefix + "o"], rt.status)
        self.decays = torch.tensor(self.decay, dtype=torch.float32, device=rt.device)
        self.norm_weight = torch.ones(self.v_dim, dtype=torch.float32, device=rt.device)
        self.freq = None
        if self.position is not None:
            self.position.load(tensors, rt)
            if self.position.rotary_dim:
                if not hasattr(self.position, "frequencies64") or getattr(self.position, "pairing", "half") != "half" \
                        or getattr(self.position, "magnitude", 1.0) != 1.0:
                    raise ConfigError("unsupported", "retention takes a half-split rotation with 64-bit frequencies")
                if self.position.rotary_dim > self.head_dim:
                    raise ConfigError("data_error", "retention: the rotated part is larger than a head")
                self.freq = self.position.frequencies64()

    def forward(self, x, ctx, cache, owns_cache=True):
        (state,) = cache
        T, H, d, dv = x.shape[0], self.heads, self.head_dim, self.v_dim
        proj = self.proj.f32(x)
        o = torch.empty((T, H, dv), dtype=torch.float32, device=x.device)
        ops.linear_scan(ops.SCAN_RETENTION, self._band(proj, "q"), self._band(proj, "k"), self._band(proj, "v"),
                        self.decays, state.state, o, ctx.q_start, ctx.slots, ctx.token_seq, positions=ctx.positions,
                        freq=self.freq, k_scale=d ** -0.5)
        return self._finish(o, self._band(proj, "g"), ctx)


@register_mixer("mlstm")
class MLSTM(_StateMixer):
    """The matrix memory of xLSTM.  q = W_q x * head_dim^-1/2, k = W_k x (heads x head_dim), v = W_v x (heads x v_dim); per
    head the logarithms of an input gate i = c tanh((W_i x + b_i) / c) and of a forget gate
    f = log sigmoid(c tanh((W_f x + b_f) / c)), c = gate_cap; per head and token, with the state S, n and m zero at first

        m' = max(f + m, i);   S = exp(f + m - m') S + exp(i - m') k v^T;   n likewise with k alone;
        o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)

    then each head's o / sqrt(mean(o^2) + eps), all heads times norm, times sigmoid(W_g x), and the output projection.
    S, n and m are the request's state, 32-bit; the gates, the recurrence, the norm and the read-out are 32-bit.

    Single tokens and portions of fewer than PORTION tokens take one kernel, token after token; longer portions are cut into
    chunks whose rows are computed side by side from the states ahead of them (csrc/mlstm.cu).

    params: hidden, heads, head_dim, v_dim, gate_cap, eps.  Tensors: <prefix>q, k [heads*head_dim, hidden]; v, g
    [heads*v_dim, hidden]; i, f [heads, hidden]; i.b, f.b [heads]; norm [heads*v_dim]; o [hidden, heads*v_dim]."""

    def __init__(self, spec, prefix=""):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden, self.heads, self.head_dim, self.v_dim = p["hidden"], p["heads"], p["head_dim"], p["v_dim"]
        self.cap, self.eps = float(p["gate_cap"]), float(p["eps"])
        if not (self.cap > 0.0):
            raise ConfigError("data_error", "mlstm: gate_cap must be positive")

    def cache_needs(self):
        H, d, dv = self.heads, self.head_dim, self.v_dim
        return (SlotState((H, d, dv)), SlotState((H, d)), SlotState((H,)))

    PORTION = 16

    def plan_key(self):
        return ("mlstm.chunks", self.PORTION)

    def plan(self, batch: HostBatch) -> Plan:
        """portions [L, 4] = (first row, tokens, slot, first chunk) of the entries of at least PORTION tokens, chunks [N, 2]
        = (first row, tokens) of theirs; short_slots: the slot of every other entry, -1 for the portions."""
        portions, chunks, short_slots = [], [], []
        for i, n in enumerate(batch.counts):
            if n < self.PORTION:
                short_slots.append(batch.slots[i])
                continue
            short_slots.append(-1)
            first = batch.q_start[i]
            portions.append((first, n, batch.slots[i], len(chunks)))
            chunks += [(first + at, min(ops.MLSTM_CHUNK, n - at)) for at in range(0, n, ops.MLSTM_CHUNK)]
        return Plan(arrays={"portions": np.asarray(portions, dtype=np.int32).reshape(-1, 4),
                            "chunks": np.asarray(chunks, dtype=np.int32).reshape(-1, 2),
                            "short_slots": np.asarray(short_slots, dtype=np.int32)},
                    values={"long": bool(portions), "short": len(portions) < len(batch.counts)})

    def tensor_specs(self):
        p, e, H, d, dv = self.prefix, self.hidden, self.heads, self.head_dim, self.v_dim
        return [TensorSpec(p + "q", (H * d, e)), TensorSpec(p + "k", (H * d, e)), TensorSpec(p + "v", (H * dv, e)),
                TensorSpec(p + "g", (H * dv, e)), TensorSpec(p + "i", (H, e)), TensorSpec(p + "f", (H, e)),
                TensorSpec(p + "i.b", (H,), wide=True), TensorSpec(p + "f.b", (H,), init="one_plus_normal", wide=True),
                TensorSpec(p + "norm", (H * dv,), init="one_plus_normal", wide=True), TensorSpec(p + "o", (e, H * dv))]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        p = self.prefix
        # (rows of zeros fill the matrix up to a multiple of 8, which the tensor-core kernels want)
        rows = self.heads * (2 * self.head_dim + 2 * self.v_dim + 2)
        pad = -rows % 8
        if pad:
            tensors = dict(tensors, **{p + "pad": torch.zeros((pad, self.hidden), dtype=tensors[p + "q"].dtype,
                                                              device=tensors[p + "q"].device)})
        self._project(tensors, ["q", "k", "v", "g", "i", "f"] + (["pad"] if pad else []), rt)
        f32 = lambda n: tensors[p + n].to(torch.float32).contiguous()
        self.i_bias, self.f_bias, self.norm_weight = f32("i.b"), f32("f.b"), f32("norm")
        self.o = Linear(tensors[p + "o"], rt.status)
        # longer portions of a bfloat16 engine: q, k, v and g in 16 bits from one product, the gates' logits in 32 from
        # another, and the chunks' products on the tensor cores
        gates = self.columns["i"][0]
        self.starts = {n: at if at < gates else at - gates for n, (at, _) in self.columns.items()}
        self.wide = self.narrow = None
        if self.proj.weight.dtype == torch.bfloat16 and self.head_dim % 8 == 0 and self.v_dim % 8 == 0:
            self.wide, self.narrow = self.proj.rows(0, gates), self.proj.rows(gates, self.proj.out_features)

    def forward(self, x, ctx, cache, owns_cache=True):
        memory, key_sum, level = cache
        gates = self.columns["i"][0]
        plan = ctx.plans.get(self.plan_key())
        portions = plan is not None and plan.long
        if portions and self.wide is not None and not self.proj.small(x):
            qkvg, logits = self.wide(x, torch.bfloat16), self.narrow.f32(x)
        else:
            proj = self.proj.f32(x)
            qkvg, logits = proj[:, :gates], proj[:, gates:]
        y = torch.empty((x.shape[0], self.heads * self.v_dim), dtype=self.rt.dtype, device=x.device)
        args = (qkvg, logits, self.starts, self.i_bias, self.f_bias, self.norm_weight, memory.state, key_sum.state,
                level.state, y)
        numbers = (self.cap, self.head_dim ** -0.5, self.eps)
        if not portions or plan.short:
            ops.mlstm_step(*args, ctx.q_start, plan.short_slots if portions else ctx.slots, *numbers)
        if portions:
            ops.mlstm_portions(*args, plan.portions, plan.chunks, *numbers)
        return self.o.f32_sums(y)
