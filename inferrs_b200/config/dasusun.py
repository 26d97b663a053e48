"""Typed configuration of the Dasusun decoder.

config.json gives every size and every constant that differs between models of the design:

    architecture   "Dasusun"
    vocab, width
    norm           {"eps": ...}: every norm of the model
    canon          {"taps": ...}: the short convolution in front of every mixer
    layers         a list; every entry has "type" (which mixer), "mixer" (its sizes and constants) and "mlp"
                   ({"kind": "dense", "ff": ...}, or null for a layer without a feed-forward)
    max_positions  optional: the most positions of a sequence

The one mixer is "latent_attention": heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims, optional scaling
{factor, original, fast, slow}}, optional mask {size} (absent: every earlier token is seen).

A key that a part needs and that is absent is an error: no size stands in code.  Keys that this reader does not know
inside `norm`, `canon`, a layer, its mixer or its feed-forward are an error too, so that a variant of the design is
refused instead of being run as this one; an unknown key at the top (a seed, a name) is named on standard error and
ignored.  A layer without a feed-forward has no second sub-layer; where the weight files hold its norms or its scale all
the same, they are read and do nothing.
"""
from __future__ import annotations

import sys
from dataclasses import dataclass, replace
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, RawConfig
from .sefalorn import _freeze, _keys, _number, _positive_ints, _thaw

DEFAULT_MAX_POSITIONS = 131072

MIXER_KEYS = {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot"}
SCALING_KEYS = {"factor", "original", "fast", "slow"}


@dataclass(frozen=True)
class DasusunLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]        # the mixer's sizes and constants, as sorted (key, value) pairs
    ff: Optional[int]                         # inner size of the feed-forward; None: the layer has none
    idle: Tuple[str, ...] = ()                # tensors of the second sub-layer that a layer without one brings anyway

    def get(self, key: str, default=None):
        return _thaw(dict(self.mixer).get(key, default))


@dataclass(frozen=True)
class DasusunConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    canon_taps: int
    layers: Tuple[DasusunLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @classmethod
    def from_raw(cls, raw: RawConfig) -> "DasusunConfig":
        src = raw.source
        known = {"architecture", "architectures", "model_type", "vocab", "width", "max_positions", "norm", "canon",
                 "layers", "eos_token_id"}
        extra = sorted(k for k in raw.values if k not in known)
        if extra:
            print(f"[inferrs_b200] {src}: keys {extra} are not part of a Dasusun configuration and are ignored",
                  file=sys.stderr)
        missing = [k for k in ("vocab", "width", "norm", "canon", "layers") if not raw.has(k)]
        if missing:
            raise ConfigError(f"{src}: Dasusun config lacks the keys {missing}")
        vocab, width = raw.get_int("vocab"), raw.get_int("width")
        max_positions = raw.get_int("max_positions", DEFAULT_MAX_POSITIONS)
        for k, v in (("vocab", vocab), ("width", width), ("max_positions", max_positions)):
            if v <= 0:
                raise ConfigError(f"{src}: key '{k}' must be positive, got {v}")
        norm = raw.values["norm"]
        if not isinstance(norm, dict) or set(norm) != {"eps"}:
            raise ConfigError(f"{src}: key 'norm' must be an object with 'eps', got {norm!r}")
        eps = _number(src, "norm.eps", norm["eps"], float)
        if eps <= 0:
            raise ConfigError(f"{src}: norm.eps must be positive, got {eps}")
        canon = raw.values["canon"]
        if not isinstance(canon, dict) or set(canon) != {"taps"} or _number(src, "canon.taps", canon["taps"], int) <= 0:
            raise ConfigError(f"{src}: key 'canon' must be an object with a positive 'taps', got {canon!r}")
        layers_raw = raw.get_list("layers")
        if not layers_raw:
            raise ConfigError(f"{src}: key 'layers' must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(entry, dict) or set(entry) - {"type", "mixer", "mlp"} or "type" not in entry \
                    or not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"{src}: {where} must be an object with 'type', 'mixer' and 'mlp', got {entry!r}")
            if entry["type"] != "latent_attention":
                raise ConfigError(f"{src}: {where}.type '{entry['type']}' is not 'latent_attention'")
            mixer = _check_mixer(src, f"{where}.mixer", entry["mixer"])
            mlp, ff = entry.get("mlp"), None
            if mlp is not None:
                if not isinstance(mlp, dict) or set(mlp) != {"kind", "ff"} or mlp["kind"] != "dense" \
                        or _number(src, f"{where}.mlp.ff", mlp["ff"], int) <= 0:
                    raise ConfigError(f"{src}: {where}.mlp must be null or of kind 'dense' with a positive 'ff', got {mlp!r}")
                ff = mlp["ff"]
            layers.append(DasusunLayer(type=entry["type"], mixer=_freeze(mixer), ff=ff))
        eos = raw.values.get("eos_token_id")
        eos_ids = () if eos is None else tuple(eos) if isinstance(eos, list) else (eos,)
        if any(isinstance(t, bool) or not isinstance(t, int) or not 0 <= t < vocab for t in eos_ids):
            raise ConfigError(f"{src}: eos_token_id must be token ids inside the vocabulary, got {eos!r}")
        return cls(vocab=vocab, width=width, max_positions=max_positions, norm_eps=eps, canon_taps=int(canon["taps"]),
                   layers=tuple(layers), eos_token_ids=eos_ids)

    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "DasusunConfig":
        """The configuration with what only the weight files say: which tensors of a second sub-layer a layer without
        a feed-forward still brings."""
        layers = list(self.layers)
        for i, layer in enumerate(layers):
            if layer.ff is None:
                idle = tuple(n for n in ("norm2", "norm2b", "ls2") if f"l{i}.{n}" in shapes)
                layers[i] = replace(layer, idle=idle)
        return replace(self, layers=tuple(layers))


def _check_mixer(src: str, where: str, given) -> Dict[str, Any]:
    out = _keys(src, where, given, MIXER_KEYS, {"mask"})
    _positive_ints(src, where, out, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
    _number(src, f"{where}.scale", out["scale"], float)
    mask = out.get("mask")
    if mask is not None and (not isinstance(mask, dict) or set(mask) != {"size"}
                             or _number(src, f"{where}.mask.size", mask["size"], int) <= 0):
        raise ConfigError(f"{src}: {where}.mask must be an object with a positive 'size', got {mask!r}")
    rot = out["rot"]
    if not isinstance(rot, dict) or not {"base", "dims"} <= set(rot) or set(rot) - {"base", "dims", "scaling"} \
            or not _number(src, f"{where}.rot.base", rot["base"], float) > 1 \
            or _number(src, f"{where}.rot.dims", rot["dims"], int) <= 0 or rot["dims"] % 2 or rot["dims"] > out["rot_dim"]:
        raise ConfigError(f"{src}: {where}.rot must give a 'base' above 1 and even 'dims' of at most rot_dim, got {rot!r}")
    scaling = rot.get("scaling")
    if scaling is not None and (not isinstance(scaling, dict) or set(scaling) != SCALING_KEYS or
                                any(not _number(src, f"{where}.rot.scaling.{k}", scaling[k], float) > 0
                                    for k in SCALING_KEYS)):
        raise ConfigError(f"{src}: {where}.rot.scaling must give positive {sorted(SCALING_KEYS)}, got {scaling!r}")
    return out
