"""Typed configuration of the Rimidra decoder, read from its config.json.

The file names the design in ``architecture`` and lists the layers one by one: each entry has ``type``
(its mixer: "attention" or "retention"), the mixer's sizes and constants in ``mixer``, and its feed-forward
in ``mlp`` (``kind`` "dense" or "moe", or null for a layer without one).  An entry with ``weights_of``: j
uses layer j's tensors (and says the rest of layer j's entry again) with a cache or state of its own.
``norm.eps`` is the one epsilon of every norm, ``vocab`` and ``width`` are the table's sizes.  An attention
without ``mask`` sees every earlier token, one without ``q_temp`` has no query temperature, a retention
without ``rot`` no rotation, a mixture without ``shared`` no shared expert.  Every size and constant is
taken from the file; a key this engine does not know inside a layer is reported on standard error and
ignored.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .model_config import ConfigError
from .tekenex_config import _int, _num, _only


@dataclass(frozen=True)
class SlopedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]                          # None: every earlier key is seen
    q_temp: Optional[Tuple[float, float]]          # (coef, every)


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[Tuple[float, int]]               # (base, dims)


@dataclass(frozen=True)
class RimidraMlpConfig:
    kind: str                                      # "dense" | "moe"
    ff: int                                        # of the dense feed-forward, or of an expert
    experts: int = 0
    top: int = 0
    shared_ff: Optional[int] = None                # None: no shared expert


@dataclass(frozen=True)
class RimidraLayerConfig:
    type: str
    mixer: Union[SlopedAttentionConfig, RetentionConfig]
    mlp: Optional[RimidraMlpConfig]
    weights_of: Optional[int] = None               # the layer whose tensors this one uses


def _object(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _attention(m: dict, where: str) -> SlopedAttentionConfig:
    _only(m, ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "q_temp"), where)
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {kv} kv_heads")
    window = temp = None
    if m.get("mask") is not None:
        mk = _object(m, "mask", where)
        _only(mk, ("size",), where + ".mask")
        window = _int(mk, "size", where + ".mask")
    if m.get("q_temp") is not None:
        t = _object(m, "q_temp", where)
        _only(t, ("coef", "every"), where + ".q_temp")
        temp = (_num(t, "coef", where + ".q_temp"), _num(t, "every", where + ".q_temp"))
        if temp[1] <= 0:
            raise ConfigError(f"config.json: {where}.q_temp.every must be positive, got {temp[1]}")
    return SlopedAttentionConfig(heads, kv, _int(m, "dim", where), _int(m, "vdim", where), _num(m, "scale", where),
                                 window, temp)


def _retention(m: dict, where: str) -> RetentionConfig:
    _only(m, ("heads", "dim", "vdim", "decay", "rot"), where)
    heads, dim = _int(m, "heads", where), _int(m, "dim", where)
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != heads \
            or not all(isinstance(g, (int, float)) and not isinstance(g, bool) and 0 < g <= 1 for g in decay):
        raise ConfigError(f"config.json: {where}.decay must list one number in (0, 1] for each of the {heads} heads")
    rot = None
    if m.get("rot") is not None:
        r = _object(m, "rot", where)
        _only(r, ("base", "dims"), where + ".rot")
        rot = (_num(r, "base", where + ".rot"), _int(r, "dims", where + ".rot"))
        if rot[1] % 2 or rot[1] > dim:
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most {dim}, got {rot[1]}")
        if rot[0] <= 0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive, got {rot[0]}")
    return RetentionConfig(heads, dim, _int(m, "vdim", where), tuple(float(g) for g in decay), rot)


def _mlp(f, where: str) -> Optional[RimidraMlpConfig]:
    if f is None:
        return None
    if not isinstance(f, dict):
        raise ConfigError(f"config.json: {where} must be an object or null")
    kind = f.get("kind")
    if kind == "dense":
        _only(f, ("kind", "ff"), where)
        return RimidraMlpConfig("dense", _int(f, "ff", where))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not known (known: dense, moe)")
    _only(f, ("kind", "router", "expert", "shared"), where)
    r, ex = _object(f, "router", where), _object(f, "expert", where)
    _only(r, ("experts", "top"), where + ".router")
    _only(ex, ("ff",), where + ".expert")
    experts, top = _int(r, "experts", where + ".router"), _int(r, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"config.json: {where}.router picks {top} of {experts} experts")
    shared = None
    if f.get("shared") is not None:
        sh = _object(f, "shared", where)
        _only(sh, ("ff",), where + ".shared")
        shared = _int(sh, "ff", where + ".shared")
    return RimidraMlpConfig("moe", _int(ex, "ff", where + ".expert"), experts, top, shared)


def _layer(entries: list, i: int) -> RimidraLayerConfig:
    e, where = entries[i], f"layers[{i}]"
    if not isinstance(e, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    _only(e, ("type", "mixer", "mlp", "weights_of"), where)
    kind, m = e.get("type"), _object(e, "mixer", where)
    if kind == "attention":
        mixer = _attention(m, where + ".mixer")
    elif kind == "retention":
        mixer = _retention(m, where + ".mixer")
    else:
        raise ConfigError(f"config.json: {where}.type {kind!r} is not known (known: attention, retention)")
    return RimidraLayerConfig(kind, mixer, _mlp(e.get("mlp"), where + ".mlp"))


def _owner(entries: list, i: int) -> Optional[int]:
    """The layer whose tensors layer i uses (None: its own)."""
    j, seen = i, set()
    while isinstance(entries[j], dict) and entries[j].get("weights_of") is not None:
        k = entries[j]["weights_of"]
        if isinstance(k, bool) or not isinstance(k, int) or not 0 <= k < len(entries) or k in seen or k == i:
            raise ConfigError(f"config.json: layers[{j}].weights_of must name another layer that leads to one with tensors "
                              f"of its own, got {k!r}")
        seen.add(k)
        j = k
    return j if j != i else None


@dataclass(frozen=True)
class RimidraConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[RimidraLayerConfig, ...]
    max_position_embeddings: int
    eos_token_ids: tuple = ()
    bos_token_id: Optional[int] = None

    @staticmethod
    def from_dict(d: dict) -> "RimidraConfig":
        norm = d.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json: 'norm' (with 'eps') is missing")
        eps = _num(norm, "eps", "norm")
        if eps < 0:
            raise ConfigError(f"config.json: norm.eps must not be negative, got {eps}")
        entries = d.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        own = [_layer(entries, i) for i in range(len(entries))]
        layers = []
        for i, lc in enumerate(own):
            j = _owner(entries, i)
            if j is not None and own[j] != lc:
                raise ConfigError(f"config.json: layers[{i}] uses the weights of layer {j} but differs from it")
            layers.append(RimidraLayerConfig(lc.type, lc.mixer, lc.mlp, j))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(x) for x in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return RimidraConfig(vocab=_int(d, "vocab", "config"), width=_int(d, "width", "config"), eps=eps,
                             layers=tuple(layers), max_position_embeddings=int(d.get("max_position_embeddings", 1 << 17)),
                             eos_token_ids=eos_ids, bos_token_id=d.get("bos_token_id"))
