"""Dense gated feed-forward."""
from __future__ import annotations

import torch

from ..csrc import ops
from ..weights.loader import TensorSpec
from .base import FeedForward
from .linear import Linear, SMS
from .registry import register_feed_forward


# Up to so many rows the package's product with the activation in its epilogue is faster than the library's
# product followed by the activation kernel (measured at 18944 x 3584: 776 against 803 us at 4,096 rows,
# 1,261 against 1,203 us at 6,144).
FUSED_ROWS = 4096


def fused_gate_up_pays(rows: int, out_features: int) -> bool:
    """Whether the package's product with the activation in its epilogue is at least as fast as the library's
    product followed by the activation kernel, for this many rows and 2 x intermediate output features.

    Measured on B200 at the 7B, 14B and 32B widths, CUDA events, cold L2.  Up to 128 rows the two are equal (the
    kernel for up to 64 rows is another matter and is not asked about here).  From 129 to 511 rows the package's
    kernel works on tiles of 128 rows, which wait for their operands a third of the time: the library is up to 36 %
    faster (14B, 384 rows: 124 against 91 us).  From 512 rows on its tiles are 256 x 256 and it is as fast as the
    library where those tiles fill whole rounds over the SMs and the rows fill the tiles (7B 768 rows: 149.5
    against 148.3 us; 14B 1,024: 197.7 / 195.5; 2,048: 369.6 / 375.8), and up to 55 % slower where they do not
    (14B 544 rows, 324 tiles of which the last third is nearly empty: 185.5 against 119.9 us)."""
    if rows <= 128:
        return True
    if rows < 512 or rows > FUSED_ROWS:
        return False
    row_tiles, col_tiles = -(-rows // 256), -(-out_features // 256)
    tiles = row_tiles * col_tiles
    rounds = -(-tiles // SMS)
    return (tiles / (rounds * SMS)) * (rows / (row_tiles * 256)) >= 0.9


@register_feed_forward("swiglu")
class SwiGLU(FeedForward):
    """down(silu(gate(x)) * up(x)) with silu(x) = x / (1 + exp(-x)), no biases
    (AIR: src/reference/reference_executor.cpp:33-35, 394-408).
    params: hidden, intermediate.  Tensors: <prefix>{gate,up}_proj.weight [intermediate, hidden],
    <prefix>down_proj.weight [hidden, intermediate].  gate and up become one matrix at load, so
    the input is read once: blocks of gate rows and of up rows for the same outputs in turn (the
    block is the largest of 128, 64, 32 that divides `intermediate`, else all of it), so that a
    tile of the product holds both factors of its outputs and the tcgen05 kernel can apply the
    activation in its epilogue, for few rows and for many; where that kernel does not apply (32-bit
    weights, an odd width) the library's product is followed by the activation kernel, which reads
    the same arrangement."""

    graph_safe = True

    ACT = ops.SILU          # the gated activation (ops.gemm_tc)
    # what follows the prefix in the names of the three matrices
    NAMES = {"gate": "gate_proj.weight", "up": "up_proj.weight", "down": "down_proj.weight"}

    def tensor_specs(self):
        e, i, p, n = self.spec["hidden"], self.spec["intermediate"], self.prefix, self.NAMES
        return [TensorSpec(p + n["gate"], (i, e)), TensorSpec(p + n["up"], (i, e)), TensorSpec(p + n["down"], (e, i))]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        p = self.prefix
        g, u = tensors[p + self.NAMES["gate"]], tensors[p + self.NAMES["up"]]
        if g.dtype != u.dtype:
            raise ValueError(f"{p}: gate and up projections are stored in different precisions")
        inter = self.intermediate = self.spec["intermediate"]
        block = next((b for b in (128, 64, 32) if inter % b == 0), inter)
        if g.dtype != torch.bfloat16:
            block = inter
        self.block = block
        if block == inter:
            w = torch.cat([g, u], dim=0)
        else:
            w = torch.stack([g.view(inter // block, block, -1), u.view(inter // block, block, -1)], dim=1)
            w = w.reshape(2 * inter, -1)
        self.gate_up = Linear(w.contiguous(), rt.status, gate_up_block=block if block != inter else 0)
        self.down = Linear(tensors[p + self.NAMES["down"]], rt.status)

    def accepts_prenormed(self, ctx, owns_cache=True):
        return self.rt.dtype == torch.bfloat16 and self.gate_up.takes_prenormed(ctx.num_tokens, silu=True)

    def forward(self, x, ctx):
        if (self.gate_up.gate_up_block and self.gate_up.tc_ok and x.dtype == torch.bfloat16
                and (self.gate_up.small(x) or fused_gate_up_pays(x.shape[0], self.gate_up.out_features))):
            # few rows or many: the tcgen05 product with SiLU(gate) * up in its epilogue (the 2 I wide
            # intermediate is never written)
            act = self.gate_up.silu_mul(x, act=self.ACT)
        else:
            gu = self.gate_up(x, torch.float32 if self.rt.is_fp32 else self.rt.dtype)
            act = torch.empty((x.shape[0], self.intermediate), dtype=self.rt.dtype, device=x.device)
            ops.silu_mul(gu, act, block=self.block, relu=self.ACT is ops.RELU)
        if self.down.small(act):
            return self.down.partial(act)
        residual = getattr(ctx, "residual", None)
        if self.down.adds_into(act, residual):
            return self.down.add_into(act, residual)
        return self.down(act, torch.float32)


@register_feed_forward("reglu")
class ReGLU(SwiGLU):
    """down(max(gate(x), 0) * up(x)): a gated feed-forward with the rectifier in SiLU's place.  params: hidden, intermediate.
    Tensors: <prefix>gate, up [intermediate, hidden], down [hidden, intermediate].  Everything else is SwiGLU's."""

    ACT = ops.RELU
    NAMES = {"gate": "gate", "up": "up", "down": "down"}


@register_feed_forward("clamped_glu")
class ClampedGLU(SwiGLU):
    """down(g * sigmoid(alpha * g) * (u + 1)) with g = min(gate(x), limit) and u = clamp(up(x), -limit, limit): a
    gated feed-forward whose gate is cut from above, whose linear branch is cut on both sides and shifted by one,
    and whose sigmoid is sharpened by alpha (1.702 gives the sigmoid form of GELU).
    params: hidden, intermediate, limit, alpha.  Tensors: <prefix>gate, up [intermediate, hidden], down
    [hidden, intermediate].  gate and up are one matrix as in SwiGLU, and as there the tcgen05 product applies the
    activation in its epilogue, for few rows and for many; where that kernel does not apply, the library's product is
    followed by the activation kernel, which reads the same arrangement."""

    NAMES = {"gate": "gate", "up": "up", "down": "down"}

    def accepts_prenormed(self, ctx, owns_cache=True):
        return False

    def forward(self, x, ctx):
        shape = (float(self.spec.get("alpha", 1.702)), float(self.spec["limit"]), 1.0)      # alpha, limit, shift
        if (self.gate_up.gate_up_block and self.gate_up.tc_ok and x.dtype == torch.bfloat16
                and (self.gate_up.small(x) or fused_gate_up_pays(x.shape[0], self.gate_up.out_features))):
            act = self.gate_up.silu_mul(x, act=shape)
        else:
            gu = self.gate_up(x, torch.float32 if self.rt.is_fp32 else self.rt.dtype)
            act = torch.empty((x.shape[0], self.intermediate), dtype=self.rt.dtype, device=x.device)
            ops.glu(gu, act, block=self.block, alpha=shape[0], limit=shape[1], shift=shape[2])
        return self.down.f32_sums(act)


@register_feed_forward("polynorm_mlp")
class PolyNormMLP(FeedForward):
    """down(act(up(x) + b_up)) + b_down with act = PolyNorm: y_i = a z_i / r1 + b z_i^2 / r2 + c z_i^3 / r3 + e with r_p = sqrt(mean_i(z_i^(2p)) + eps)
    over the `intermediate` columns of one row, and (a, b, c, e) the four numbers of the tensor act.  params: hidden, intermediate, eps.  Tensors: <prefix>up [intermediate, hidden], up.b
    [intermediate], down [hidden, intermediate], down.b [hidden], act [4].

    z leaves the first product in 32-bit; one kernel adds b_up, takes the three norms and writes the activation in the
    compute dtype.  b_down rides in the second product: the matrix gets one more column that holds it (and zeros up
    to a multiple of 8 columns), the activation a matching column of ones."""

    graph_safe = True

    def tensor_specs(self):
        e, f, p = self.spec["hidden"], self.spec["intermediate"], self.prefix
        return [TensorSpec(p + "up", (f, e)), TensorSpec(p + "up.b", (f,), wide=True), TensorSpec(p + "down", (e, f)),
                TensorSpec(p + "down.b", (e,), wide=True),
                TensorSpec(p + "act", (4,), init="one_plus_normal", std=0.3, wide=True)]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        p = self.prefix
        self.intermediate, self.eps = self.spec["intermediate"], float(self.spec["eps"])
        self.up = Linear(tensors[p + "up"], rt.status)
        self.up_bias = tensors[p + "up.b"].to(torch.float32).contiguous()
        down = tensors[p + "down"]
        f = self.intermediate
        self.padded = (f // 8 + 1) * 8
        w = torch.zeros((down.shape[0], self.padded), dtype=down.dtype, device=down.device)
        w[:, :f] = down
        w[:, f] = tensors[p + "down.b"].to(down.dtype)
        self.down = Linear(w, rt.status)
        self.coefficients = tuple(float(v) for v in tensors[p + "act"].to(torch.float32).cpu().tolist())

    def forward(self, x, ctx):
        z = self.up.f32(x)
        act = torch.empty((x.shape[0], self.padded), dtype=self.rt.dtype, device=x.device)
        ops.polynorm(z, self.up_bias, self.coefficients, self.eps, act, self.intermediate)
        return self.down.f32_sums(act)


@register_feed_forward("relu2_mlp")
class Relu2MLP(FeedForward):
    """down(max(up(x), 0)^2): one hidden layer without a gate and without biases, whose activation is the square of
    the rectifier.  params: hidden, intermediate.  Tensors: <prefix>up [intermediate, hidden], down [hidden,
    intermediate].

    In bfloat16 the tcgen05 product squares the rectified sums in its epilogue (32-bit, rounded once), for few rows and
    for as many as that kernel is at least as fast as the library's (fused_gate_up_pays); else the library's product is
    followed by the kernel that squares the rectified values (from 32-bit sums in a float32 engine)."""

    graph_safe = True

    def tensor_specs(self):
        e, f, p = self.spec["hidden"], self.spec["intermediate"], self.prefix
        return [TensorSpec(p + "up", (f, e)), TensorSpec(p + "down", (e, f))]

    def load(self, tensors, rt):
        super().load(tensors, rt)
        self.intermediate = self.spec["intermediate"]
        self.up = Linear(tensors[self.prefix + "up"], rt.status)
        self.down = Linear(tensors[self.prefix + "down"], rt.status)

    def forward(self, x, ctx):
        if self.up.tc_ok and x.dtype == torch.bfloat16 and (self.up.small(x) or
                                                            fused_gate_up_pays(x.shape[0], self.up.out_features)):
            act = self.up.relu2(x)
        else:
            z = self.up(x, torch.float32 if self.rt.is_fp32 else self.rt.dtype)
            act = ops.relu2(z, torch.empty(z.shape, dtype=self.rt.dtype, device=x.device))
        return self.down.f32_sums(act)
