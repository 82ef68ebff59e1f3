"""Typed configuration of the Sesulorn decoder, read from config.json's own keys.

config.json names the design under "architecture" and gives "vocab", "width", "norm" {"eps"}, "loop" {"start", "stop",
"times"} (the layers start .. stop - 1 run `times` times over; may be absent) and "layers": every entry has a "type"
("attention", "channel_delta" or "latent_attention"), the mixer's sizes and constants under "mixer" and its feed-forward
under "mlp" (null: none; kind "dense" or "moe").  Every size and constant that may differ between two models of the design
is read from there.  Three sizes of a mixer are only the shapes of its tensors: the rows of an attention layer's distance
table, and the narrow middles of a channel_delta layer's decay and gate.  Where there is no model file (random weights) they
are the mixer's keys "buckets", "decay_rank" and "gate_rank".
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple

from .bivizen_config import _get
from .model_config import ConfigError

MIXER_TYPES = ("attention", "channel_delta", "latent_attention")
# No key of config.json bounds a request's length; the block tables need a width, and this is it.
POSITIONS = 1 << 20


@dataclass(frozen=True)
class SesulornFeedForward:
    """kind "dense": a gated feed-forward of width ff with SiLU.  kind "moe": `experts` experts of width ff with the clamped
    activation (`limit`), of which a token takes `top` out of the `keep` best of `groups` groups; a shared expert of width
    shared_ff (0: none) with a limit of its own beside them."""
    kind: str
    ff: int
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0
    shared_limit: float = 0.0


@dataclass(frozen=True)
class SesulornLayer:
    type: str
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0            # attention, channel_delta
    scale: float = 0.0           # attention, latent_attention
    bias_max: float = 0.0        # attention: the distance from which the table's last row serves
    buckets: int = 0             # attention: rows of the distance table
    conv: int = 0                # channel_delta: taps
    decay_rank: int = 0          # channel_delta
    gate_rank: int = 0           # channel_delta
    q_rank: int = 0              # latent_attention
    kv_rank: int = 0             # latent_attention
    rot_dim: int = 0             # latent_attention
    rot_base: float = 1.0        # latent_attention
    mlp: Optional[SesulornFeedForward] = None


def _feed_forward(f: Mapping[str, Any], where: str) -> SesulornFeedForward:
    kind = _get(f, "kind", str, where)
    if kind == "dense":
        return SesulornFeedForward(kind="dense", ff=_get(f, "ff", int, where))
    if kind != "moe":
        raise ConfigError("unsupported", f"{where}: feed-forward kind {kind!r} (known: dense, moe)")
    e, r, shared = f.get("expert"), f.get("router"), f.get("shared")
    g = r.get("groups") if isinstance(r, Mapping) else None
    return SesulornFeedForward(
        kind="moe", ff=_get(e, "ff", int, where + ".expert"), limit=_get(e, "limit", float, where + ".expert"),
        experts=_get(r, "experts", int, where + ".router"), top=_get(r, "top", int, where + ".router"),
        groups=_get(g, "count", int, where + ".router.groups") if g is not None else 1,
        keep=_get(g, "keep", int, where + ".router.groups") if g is not None else 1,
        shared_ff=_get(shared, "ff", int, where + ".shared") if shared is not None else 0,
        shared_limit=_get(shared, "limit", float, where + ".shared") if shared is not None else 0.0)


@dataclass(frozen=True)
class SesulornConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    loop_start: int
    loop_stop: int
    loop_times: int
    has_loop: bool               # config.json has "loop" (and the model file its matrix), even if the stretch is empty
    layers: Tuple[SesulornLayer, ...]
    max_positions: int = POSITIONS
    eos_token_id: Optional[int] = None
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False)

    reads_shapes = True

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], shapes=None) -> "SesulornConfig":
        arch = d.get("architecture") or (d.get("architectures") or [None])[0]
        if arch is None:
            raise ConfigError("data_error", "config.json lacks 'architecture'")
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("data_error", "config.json lacks 'layers'")
        layers = []
        for i, entry in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = _get(entry, "type", str, where)
            if kind not in MIXER_TYPES:
                raise ConfigError("unsupported", f"{where}: mixer type {kind!r} (known: {', '.join(MIXER_TYPES)})")
            m = entry.get("mixer")
            if not isinstance(m, Mapping):
                raise ConfigError("data_error", f"config.json lacks 'mixer' in {where}")
            wm = where + ".mixer"

            def shaped(key, tensor, typ=int):
                """A size that is a tensor's first dimension; without a model file, the mixer's key."""
                shape = None if shapes is None else shapes.get(f"l{i}.mix.{tensor}")
                return int(shape[0]) if shape else _get(m, key, typ, wm)

            kw = dict(type=kind, heads=_get(m, "heads", int, wm), dim=_get(m, "dim", int, wm), vdim=_get(m, "vdim", int, wm))
            if kind == "attention":
                kw.update(kv_heads=_get(m, "kv_heads", int, wm), scale=_get(m, "scale", float, wm),
                          bias_max=_get(m, "bias_max", float, wm), buckets=shaped("buckets", "rel"))
            elif kind == "channel_delta":
                kw.update(kv_heads=_get(m, "kv_heads", int, wm), conv=_get(m, "conv", int, wm),
                          decay_rank=shaped("decay_rank", "a1"), gate_rank=shaped("gate_rank", "g1"))
            else:
                rot_dim = _get(m, "rot_dim", int, wm)
                kw.update(scale=_get(m, "scale", float, wm), kv_rank=_get(m, "kv_rank", int, wm),
                          q_rank=_get(m, "q_rank", int, wm), rot_dim=rot_dim)
                if rot_dim:
                    rot = m.get("rot")
                    kw.update(rot_base=_get(rot, "base", float, wm + ".rot"))
                    if _get(rot, "dims", int, wm + ".rot", rot_dim, required=False) != rot_dim:
                        raise ConfigError("data_error", f"{wm}: the rotation covers the rotated part, all of it")
            if entry.get("mlp") is not None:
                kw["mlp"] = _feed_forward(entry["mlp"], where + ".mlp")
            layers.append(SesulornLayer(**kw))
        where = "config.json"
        loop = d.get("loop")
        eos = d.get("eos_token_id")
        cfg = cls(architecture=arch, vocab=_get(d, "vocab", int, where), width=_get(d, "width", int, where),
                  eps=_get(d.get("norm"), "eps", float, "norm"),
                  loop_start=_get(loop, "start", int, "loop") if loop is not None else 0,
                  loop_stop=_get(loop, "stop", int, "loop") if loop is not None else 0,
                  loop_times=_get(loop, "times", int, "loop") if loop is not None else 1,
                  has_loop=loop is not None, layers=tuple(layers),
                  max_positions=_get(d, "max_positions", int, where, POSITIONS, required=False),
                  eos_token_id=eos if isinstance(eos, int) else None, raw=dict(d))
        cfg.validate()
        return cfg

    @property
    def loops(self) -> bool:
        return self.loop_stop > self.loop_start

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m = {"heads": l.heads, "dim": l.dim, "vdim": l.vdim}
            if l.type == "attention":
                m.update(kv_heads=l.kv_heads, scale=l.scale, bias_max=l.bias_max, buckets=l.buckets)
            elif l.type == "channel_delta":
                m.update(kv_heads=l.kv_heads, conv=l.conv, decay_rank=l.decay_rank, gate_rank=l.gate_rank)
            else:
                m.update(scale=l.scale, q_rank=l.q_rank, kv_rank=l.kv_rank, rot_dim=l.rot_dim)
                if l.rot_dim:
                    m["rot"] = {"base": l.rot_base, "dims": l.rot_dim}
            f = l.mlp
            mlp = None
            if f is not None and f.kind == "dense":
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit},
                       "router": {"experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff, "limit": f.shared_limit}
            layers.append({"type": l.type, "mixer": m, "mlp": mlp})
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "layers": layers}
        if self.has_loop:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        if self.max_positions != POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("data_error", "Sesulorn geometry is incomplete: vocab and width must be positive")
        if not (self.eps > 0.0):
            raise ConfigError("data_error", "Sesulorn norm eps is missing or invalid")
        n = len(self.layers)
        if not (0 <= self.loop_start <= self.loop_stop <= n) or self.loop_times < 1:
            raise ConfigError("data_error", f"loop: 0 <= start <= stop <= {n} layers and times >= 1")
        for i, l in enumerate(self.layers):
            where = f"layers[{i}]"
            if min(l.heads, l.dim, l.vdim) <= 0:
                raise ConfigError("data_error", f"{where}: heads, dim and vdim must be positive")
            if l.type != "latent_attention" and (l.kv_heads <= 0 or l.heads % l.kv_heads):
                raise ConfigError("data_error", f"{where}: heads must be a multiple of kv_heads")
            if l.type == "attention" and (l.buckets < 2 or l.bias_max <= l.buckets // 2):
                raise ConfigError("data_error", f"{where}: the distance table needs 2 rows at least, and bias_max more than "
                                                "half of them")
            if l.type == "attention" and not (l.scale > 0.0):
                raise ConfigError("data_error", f"{where}: scale must be positive")
            if l.type == "channel_delta" and min(l.conv, l.decay_rank, l.gate_rank) <= 0:
                raise ConfigError("data_error", f"{where}: conv and the narrow middles must be positive")
            if l.type == "latent_attention" and (min(l.q_rank, l.kv_rank) <= 0 or l.rot_dim < 0 or l.rot_dim % 2):
                raise ConfigError("data_error", f"{where}: q_rank and kv_rank must be positive, rot_dim even")
            f = l.mlp
            if f is None:
                continue
            if f.ff <= 0:
                raise ConfigError("data_error", f"{where}.mlp: ff must be positive")
            if f.kind == "moe":
                if f.experts <= 0 or not (0 < f.top <= f.experts) or f.shared_ff < 0:
                    raise ConfigError("data_error", f"{where}.mlp: experts and top (at most experts) must be positive")
                if not (f.limit > 0.0) or (f.shared_ff and not (f.shared_limit > 0.0)):
                    raise ConfigError("data_error", f"{where}.mlp: limit must be positive")
                if f.groups < 1 or f.experts % f.groups or not (1 <= f.keep <= f.groups) \
                        or f.top > f.keep * (f.experts // f.groups):
                    raise ConfigError("data_error", f"{where}.mlp.router.groups: equal groups, 1 <= keep <= count, and the "
                                                    "kept groups must hold at least `top` experts")
