"""Typed configuration of the Matusun decoder, read from its config.json.

The file names the design in ``architecture`` and lists the layers one by one: each entry has ``type``
(its mixer: "attention" or "mamba1"), the mixer's sizes and constants in ``mixer``, and its feed-forward in
``mlp`` (``kind`` "moe", or null for a layer without one).  ``streams`` is the number of residual streams,
``loop`` (optional) says which layers run several times in a row, ``norm.eps`` is the one epsilon of every
norm, ``vocab`` and ``width`` are the table's sizes.  An attention without ``mask`` sees every earlier token,
one without ``rot`` has no rotation, a mixture without ``shared`` no shared expert, a router without
``identity`` no experts that hand on their input and one without ``scale`` a factor of 1.  Every size and
constant is taken from the file; a key this engine does not know inside a layer is reported on standard error
and ignored.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union

from .bevuvik_config import LoopConfig, read_loop
from .model_config import ConfigError
from .rimidra_config import _object
from .tekenex_config import _int, _num, _only


@dataclass(frozen=True)
class RowNormedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]                          # None: every earlier key is seen
    rot: Optional[Tuple[float, int]]               # (base, dims)


@dataclass(frozen=True)
class SelectiveScanConfig:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class MatusunMlpConfig:
    ff: int                                        # of an expert
    experts: int
    top: int
    identity: int                                  # router outputs past the experts that hand on their input
    scale: float                                   # factor on the experts' weights
    shared_ff: Optional[int] = None                # None: no shared expert


@dataclass(frozen=True)
class MatusunLayerConfig:
    type: str
    mixer: Union[RowNormedAttentionConfig, SelectiveScanConfig]
    mlp: Optional[MatusunMlpConfig]


def _attention(m: dict, where: str) -> RowNormedAttentionConfig:
    _only(m, ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"), where)
    heads, kv, dim = _int(m, "heads", where), _int(m, "kv_heads", where), _int(m, "dim", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {kv} kv_heads")
    window = rot = None
    if m.get("mask") is not None:
        mk = _object(m, "mask", where)
        _only(mk, ("size",), where + ".mask")
        window = _int(mk, "size", where + ".mask")
    if m.get("rot") is not None:
        r = _object(m, "rot", where)
        _only(r, ("base", "dims"), where + ".rot")
        rot = (_num(r, "base", where + ".rot"), _int(r, "dims", where + ".rot"))
        if rot[1] % 2 or rot[1] > dim:
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most {dim}, got {rot[1]}")
        if rot[0] <= 0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive, got {rot[0]}")
    return RowNormedAttentionConfig(heads, kv, dim, _int(m, "vdim", where), _num(m, "scale", where), window, rot)


def _scan(m: dict, where: str) -> SelectiveScanConfig:
    _only(m, ("inner", "state", "dt_rank", "conv"), where)
    return SelectiveScanConfig(*(_int(m, k, where) for k in ("inner", "state", "dt_rank", "conv")))


def _mlp(f, where: str) -> Optional[MatusunMlpConfig]:
    if f is None:
        return None
    if not isinstance(f, dict):
        raise ConfigError(f"config.json: {where} must be an object or null")
    if f.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}.kind {f.get('kind')!r} is not known (known: moe)")
    _only(f, ("kind", "router", "expert", "shared"), where)
    r, ex = _object(f, "router", where), _object(f, "expert", where)
    _only(r, ("experts", "top", "identity", "scale"), where + ".router")
    _only(ex, ("ff",), where + ".expert")
    experts, top = _int(r, "experts", where + ".router"), _int(r, "top", where + ".router")
    identity = r.get("identity") or 0
    if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
        raise ConfigError(f"config.json: {where}.router.identity must be an integer >= 0, got {identity!r}")
    scale = 1.0 if r.get("scale") is None else _num(r, "scale", where + ".router")
    if top > experts + identity:
        raise ConfigError(f"config.json: {where}.router picks {top} of {experts + identity} experts")
    shared = None
    if f.get("shared") is not None:
        sh = _object(f, "shared", where)
        _only(sh, ("ff",), where + ".shared")
        shared = _int(sh, "ff", where + ".shared")
    return MatusunMlpConfig(_int(ex, "ff", where + ".expert"), experts, top, identity, scale, shared)


def _layer(e, where: str) -> MatusunLayerConfig:
    if not isinstance(e, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    _only(e, ("type", "mixer", "mlp"), where)
    kind, m = e.get("type"), _object(e, "mixer", where)
    if kind == "attention":
        mixer = _attention(m, where + ".mixer")
    elif kind == "mamba1":
        mixer = _scan(m, where + ".mixer")
    else:
        raise ConfigError(f"config.json: {where}.type {kind!r} is not known (known: attention, mamba1)")
    return MatusunLayerConfig(kind, mixer, _mlp(e.get("mlp"), where + ".mlp"))


@dataclass(frozen=True)
class MatusunConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    layers: Tuple[MatusunLayerConfig, ...]
    loop: Optional[LoopConfig]
    max_position_embeddings: int
    eos_token_ids: tuple = ()
    bos_token_id: Optional[int] = None

    @staticmethod
    def from_dict(d: dict) -> "MatusunConfig":
        eps = _num(_object(d, "norm", "config"), "eps", "norm")
        if eps < 0:
            raise ConfigError(f"config.json: norm.eps must not be negative, got {eps}")
        entries = d.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = tuple(_layer(e, f"layers[{i}]") for i, e in enumerate(entries))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(x) for x in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return MatusunConfig(vocab=_int(d, "vocab", "config"), width=_int(d, "width", "config"), eps=eps,
                             streams=_int(d, "streams", "config"), layers=layers, loop=read_loop(d, len(layers)),
                             max_position_embeddings=int(d.get("max_position_embeddings", 1 << 17)),
                             eos_token_ids=eos_ids, bos_token_id=d.get("bos_token_id"))
