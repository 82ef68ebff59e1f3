"""Typed configuration of the Dafotar decoder, read from config.json's own keys.

config.json names the design under "architecture" and gives "vocab", "width", "norm" {"eps"}, "streams" (how many
residual streams stand side by side), "canon" {"taps"} (the convolution ahead of every mixer) and "layers": every entry
has a "type" ("attention" or "mlstm"), the mixer's sizes and constants under "mixer" and its feed-forward under "mlp"
(null: none; kind "dense" with "ff").  A mixer gives "heads", "dim" and "vdim"; attention also "kv_heads", "scale",
"mask" {"size"} (the window), "rot" {"base", "dims"} and, where it reads an earlier layer's keys and values, "kv_from";
mlstm its "gate_cap".  Every size and constant that may differ between two models of the design is read from there;
nothing has a default in code except keys that a model may leave out (the convolution, a window, a rotation, kv_from).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Tuple

from .bivizen_config import _get
from .model_config import ConfigError

MIXER_TYPES = ("attention", "mlstm")
# No key of config.json bounds a request's length; the block tables need a width, and this is it.
POSITIONS = 1 << 20


@dataclass(frozen=True)
class DafotarLayer:
    type: str
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0                 # attention
    scale: float = 0.0                # attention
    window: Optional[int] = None      # attention (None: every earlier key)
    rot_dims: int = 0                 # attention: the rotated part of a head of q and k
    rot_base: float = 0.0             # attention (0: no rotation, neither of q and k nor of the values)
    kv_from: Optional[int] = None     # attention: the layer whose keys and values this one reads
    gate_cap: float = 0.0             # mlstm
    ff: int = 0                       # width of the dense feed-forward (0: the layer has none)


@dataclass(frozen=True)
class DafotarConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    streams: int
    taps: int
    layers: Tuple[DafotarLayer, ...]
    max_positions: int = POSITIONS
    eos_token_id: Optional[int] = None
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "DafotarConfig":
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
            kw = dict(type=kind, heads=_get(m, "heads", int, wm), dim=_get(m, "dim", int, wm),
                      vdim=_get(m, "vdim", int, wm))
            if kind == "attention":
                kw.update(kv_heads=_get(m, "kv_heads", int, wm), scale=_get(m, "scale", float, wm),
                          kv_from=_get(m, "kv_from", int, wm, None, required=False))
                if m.get("mask") is not None:
                    kw["window"] = _get(m["mask"], "size", int, wm + ".mask")
                if m.get("rot") is not None:
                    kw.update(rot_dims=_get(m["rot"], "dims", int, wm + ".rot"),
                              rot_base=_get(m["rot"], "base", float, wm + ".rot"))
            else:
                kw["gate_cap"] = _get(m, "gate_cap", float, wm)
            f = entry.get("mlp")
            if f is not None:
                fkind = _get(f, "kind", str, where + ".mlp")
                if fkind != "dense":
                    raise ConfigError("unsupported", f"{where}.mlp: feed-forward kind {fkind!r} (known: dense)")
                kw["ff"] = _get(f, "ff", int, where + ".mlp")
                if kw["ff"] <= 0:
                    raise ConfigError("data_error", f"{where}.mlp: ff must be positive")
            layers.append(DafotarLayer(**kw))
        where = "config.json"
        eos = d.get("eos_token_id")
        cfg = cls(architecture=arch, vocab=_get(d, "vocab", int, where), width=_get(d, "width", int, where),
                  eps=_get(d.get("norm"), "eps", float, "norm"), streams=_get(d, "streams", int, where),
                  taps=_get(d["canon"], "taps", int, "canon") if d.get("canon") is not None else 0,
                  layers=tuple(layers),
                  max_positions=_get(d, "max_positions", int, where, POSITIONS, required=False),
                  eos_token_id=eos if isinstance(eos, int) else None, raw=dict(d))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m = {"heads": l.heads, "dim": l.dim, "vdim": l.vdim}
            if l.type == "attention":
                m.update(kv_heads=l.kv_heads, scale=l.scale)
                if l.window is not None:
                    m["mask"] = {"size": l.window}
                if l.rot_base:
                    m["rot"] = {"base": l.rot_base, "dims": l.rot_dims}
                if l.kv_from is not None:
                    m["kv_from"] = l.kv_from
            else:
                m["gate_cap"] = l.gate_cap
            layers.append({"type": l.type, "mixer": m, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None})
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "streams": self.streams, "layers": layers}
        if self.taps:
            d["canon"] = {"taps": self.taps}
        if self.max_positions != POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("data_error", "Dafotar geometry is incomplete: vocab and width must be positive")
        if not (self.eps > 0.0):
            raise ConfigError("data_error", "Dafotar norm eps is missing or invalid")
        if self.streams < 1 or self.taps < 0:
            raise ConfigError("data_error", "Dafotar: at least one stream, and not a negative number of taps")
        for i, l in enumerate(self.layers):
            if min(l.heads, l.dim, l.vdim) <= 0:
                raise ConfigError("data_error", f"layers[{i}]: heads, dim and vdim must be positive")
            if l.type == "mlstm":
                if not (l.gate_cap > 0.0):
                    raise ConfigError("data_error", f"layers[{i}]: gate_cap must be positive")
                continue
            if l.kv_heads <= 0 or l.heads % l.kv_heads:
                raise ConfigError("data_error", f"layers[{i}]: heads must be a multiple of kv_heads")
            if l.window is not None and l.window < 1:
                raise ConfigError("data_error", f"layers[{i}].mixer.mask: size must be positive")
            if l.rot_base and (l.rot_dims < 0 or l.rot_dims % 2 or l.rot_dims > l.dim or l.vdim % 2
                               or not (l.rot_base > 0.0)):
                raise ConfigError("data_error", f"layers[{i}].mixer.rot: dims must be even and at most dim, vdim even, "
                                                "base positive")
            if l.kv_from is not None:
                if not (0 <= l.kv_from < i) or self.layers[l.kv_from].type != "attention" \
                        or self.layers[l.kv_from].kv_from is not None:
                    raise ConfigError("data_error", f"layers[{i}].mixer.kv_from: {l.kv_from} is not an earlier attention "
                                                    "layer with keys and values of its own")
                o = self.layers[l.kv_from]
                if (o.kv_heads, o.dim, o.vdim) != (l.kv_heads, l.dim, l.vdim):
                    raise ConfigError("data_error", f"layers[{i}].mixer.kv_from: layer {l.kv_from} keeps keys and values "
                                                    "of other sizes")
