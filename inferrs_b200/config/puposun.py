"""Typed configuration of the Puposun decoder.

config.json gives every size and every constant that differs between models of the design:

    architecture   "Puposun"
    vocab, width
    norm           {"eps": ...}: every norm of the model
    embedding      {"scale": ...}: embedding rows are multiplied by it
    logit_softcap  optional: logits become cap tanh(logits / cap)
    layers         a list; every entry has "type" (which mixer), "mixer" (its sizes and constants) and "mlp"
                   (a feed-forward, or null for a layer without one)
    loop           optional {"start", "stop", "times"}: layers start .. stop - 1 run that many times in a row
    max_positions  optional: the most positions of a sequence

Mixers: "attention" (heads, kv_heads, dim, vdim, scale, optional softcap, optional rot {base, dims}) and "attention_2"
(heads, kv_heads, dim, vdim, scale, optional mask {size, keep_first}, optional rot {base, dims}).  The values are the
projected keys, so vdim is dim.  Feed-forward: {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "scale",
optional groups {count, keep}}}.

A key that the chosen part needs and that is absent is an error: no size stands in code.  Keys that this reader does
not know inside `norm`, `embedding`, `loop`, a layer, its mixer or its feed-forward are an error too, so that a variant
of the design is refused instead of being run as this one; an unknown key at the top (a seed, a name) is named on
standard error and ignored.
"""
from __future__ import annotations

import sys
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, RawConfig
from .sefalorn import _freeze, _keys, _number, _positive_ints, _thaw

DEFAULT_MAX_POSITIONS = 131072

MIXER_KEYS = {"heads", "kv_heads", "dim", "vdim", "scale"}
OPTIONAL_KEYS = {"attention": {"softcap", "rot"}, "attention_2": {"mask", "rot"}}


@dataclass(frozen=True)
class PuposunLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]            # the mixer's sizes and constants, as sorted (key, value) pairs
    mlp: Optional[Tuple[Tuple[str, Any], ...]]    # the feed-forward's; None: the layer has none

    def get(self, key: str, default=None):
        return _thaw(dict(self.mixer).get(key, default))

    def mlp_get(self, key: str, default=None):
        return None if self.mlp is None else _thaw(dict(self.mlp).get(key, default))


@dataclass(frozen=True)
class PuposunConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    embedding_scale: float
    logit_softcap: Optional[float]
    layers: Tuple[PuposunLayer, ...]
    loop: Optional[Tuple[int, int, int]] = None    # start, stop, times
    eos_token_ids: Tuple[int, ...] = ()

    @classmethod
    def from_raw(cls, raw: RawConfig) -> "PuposunConfig":
        src = raw.source
        known = {"architecture", "architectures", "model_type", "vocab", "width", "max_positions", "norm", "embedding",
                 "logit_softcap", "layers", "loop", "eos_token_id"}
        extra = sorted(k for k in raw.values if k not in known)
        if extra:
            print(f"[inferrs_b200] {src}: keys {extra} are not part of a Puposun configuration and are ignored",
                  file=sys.stderr)
        missing = [k for k in ("vocab", "width", "norm", "embedding", "layers") if not raw.has(k)]
        if missing:
            raise ConfigError(f"{src}: Puposun config lacks the keys {missing}")
        vocab, width = raw.get_int("vocab"), raw.get_int("width")
        max_positions = raw.get_int("max_positions", DEFAULT_MAX_POSITIONS)
        for k, v in (("vocab", vocab), ("width", width), ("max_positions", max_positions)):
            if v <= 0:
                raise ConfigError(f"{src}: key '{k}' must be positive, got {v}")
        eps = _single(src, raw, "norm", "eps")
        if eps <= 0:
            raise ConfigError(f"{src}: norm.eps must be positive, got {eps}")
        scale = _single(src, raw, "embedding", "scale")
        cap = raw.values.get("logit_softcap")
        if cap is not None and not _number(src, "logit_softcap", cap, float) > 0:
            raise ConfigError(f"{src}: logit_softcap must be positive, got {cap!r}")
        layers_raw = raw.get_list("layers")
        if not layers_raw:
            raise ConfigError(f"{src}: key 'layers' must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(entry, dict) or set(entry) - {"type", "mixer", "mlp"} or "type" not in entry \
                    or not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"{src}: {where} must be an object with 'type', 'mixer' and 'mlp', got {entry!r}")
            if entry["type"] not in OPTIONAL_KEYS:
                raise ConfigError(f"{src}: {where}.type '{entry['type']}' is not one of {sorted(OPTIONAL_KEYS)}")
            mixer = _check_mixer(src, f"{where}.mixer", entry["mixer"], OPTIONAL_KEYS[entry["type"]])
            mlp = _check_mlp(src, where, entry.get("mlp"))
            layers.append(PuposunLayer(type=entry["type"], mixer=_freeze(mixer), mlp=None if mlp is None else _freeze(mlp)))
        eos = raw.values.get("eos_token_id")
        eos_ids = () if eos is None else tuple(eos) if isinstance(eos, list) else (eos,)
        if any(isinstance(t, bool) or not isinstance(t, int) or not 0 <= t < vocab for t in eos_ids):
            raise ConfigError(f"{src}: eos_token_id must be token ids inside the vocabulary, got {eos!r}")
        return cls(vocab=vocab, width=width, max_positions=max_positions, norm_eps=eps, embedding_scale=scale,
                   logit_softcap=None if cap is None else float(cap), layers=tuple(layers),
                   loop=_check_loop(src, raw.values.get("loop"), len(layers)), eos_token_ids=eos_ids)


def _single(src: str, raw: RawConfig, key: str, name: str) -> float:
    """The one number of an object {name: number}."""
    v = raw.values[key]
    if not isinstance(v, dict) or set(v) != {name}:
        raise ConfigError(f"{src}: key '{key}' must be an object with '{name}', got {v!r}")
    return _number(src, f"{key}.{name}", v[name], float)


def _check_loop(src: str, loop, n_layers: int) -> Optional[Tuple[int, int, int]]:
    if loop is None:
        return None
    if not isinstance(loop, dict) or set(loop) != {"start", "stop", "times"}:
        raise ConfigError(f"{src}: key 'loop' must be an object with 'start', 'stop' and 'times', got {loop!r}")
    start, stop, times = (_number(src, f"loop.{k}", loop[k], int) for k in ("start", "stop", "times"))
    if not 0 <= start < stop <= n_layers or times < 1:
        raise ConfigError(f"{src}: the loop runs layers start .. stop - 1 of {n_layers} at least once, got {loop!r}")
    return start, stop, times


def _check_mixer(src: str, where: str, given, optional: set) -> Dict[str, Any]:
    out = _keys(src, where, given, MIXER_KEYS, optional)
    _positive_ints(src, where, out, ("heads", "kv_heads", "dim", "vdim"))
    _number(src, f"{where}.scale", out["scale"], float)
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"{src}: {where}: {out['heads']} heads are not a multiple of {out['kv_heads']} kv_heads")
    if out["vdim"] != out["dim"]:
        raise ConfigError(f"{src}: {where}: the values are the keys, so vdim {out['vdim']} must be dim {out['dim']}")
    if "softcap" in out and not _number(src, f"{where}.softcap", out["softcap"], float) > 0:
        raise ConfigError(f"{src}: {where}.softcap must be positive, got {out['softcap']!r}")
    mask = out.get("mask")
    if mask is not None and (not isinstance(mask, dict) or not {"size"} <= set(mask) <= {"size", "keep_first"}
                             or _number(src, f"{where}.mask.size", mask["size"], int) <= 0
                             or _number(src, f"{where}.mask.keep_first", mask.get("keep_first", 0), int) < 0):
        raise ConfigError(f"{src}: {where}.mask must be an object with a positive 'size' and a 'keep_first' that is not "
                          f"negative, got {mask!r}")
    rot = out.get("rot")
    if rot is not None:
        if not isinstance(rot, dict) or set(rot) != {"base", "dims"} \
                or not _number(src, f"{where}.rot.base", rot["base"], float) > 1 \
                or _number(src, f"{where}.rot.dims", rot["dims"], int) <= 0 or rot["dims"] % 2 \
                or rot["dims"] > out["dim"]:
            raise ConfigError(f"{src}: {where}.rot must give a 'base' above 1 and even 'dims' of at most the head's "
                              f"size, got {rot!r}")
    return out


def _check_mlp(src: str, where: str, mlp) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe" or set(mlp) != {"kind", "expert", "router"}:
        raise ConfigError(f"{src}: {where}.mlp must be null or an object of kind 'moe' with 'expert' and 'router', got {mlp!r}")
    expert, router = mlp["expert"], mlp["router"]
    if not isinstance(expert, dict) or set(expert) != {"ff"} \
            or _number(src, f"{where}.mlp.expert.ff", expert["ff"], int) <= 0:
        raise ConfigError(f"{src}: {where}.mlp.expert must be an object with a positive 'ff', got {expert!r}")
    need = {"experts", "top", "scale"}
    if not isinstance(router, dict) or not need <= set(router) <= need | {"groups"} \
            or not 0 < _number(src, f"{where}.mlp.router.top", router["top"], int) \
            <= _number(src, f"{where}.mlp.router.experts", router["experts"], int):
        raise ConfigError(f"{src}: {where}.mlp.router must give 'experts', 'top' and 'scale' with 0 < top <= experts, "
                          f"got {router!r}")
    _number(src, f"{where}.mlp.router.scale", router["scale"], float)
    groups = router.get("groups")
    if groups is not None:
        if not isinstance(groups, dict) or set(groups) != {"count", "keep"}:
            raise ConfigError(f"{src}: {where}.mlp.router.groups must be an object with 'count' and 'keep', got {groups!r}")
        count, keep = (_number(src, f"{where}.mlp.router.groups.{k}", groups[k], int) for k in ("count", "keep"))
        if count <= 0 or router["experts"] % count or not 0 < keep <= count \
                or keep * (router["experts"] // count) < router["top"]:
            raise ConfigError(f"{src}: {where}.mlp.router.groups: {keep} of {count} equal groups of {router['experts']} "
                              f"experts must hold the {router['top']} that are chosen")
    return {k: v for k, v in mlp.items()}
