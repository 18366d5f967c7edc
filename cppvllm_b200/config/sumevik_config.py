"""Typed configuration of the Sumevik decoder, read from its ``config.json``.

Top level: ``vocab``, ``width``, ``norm.eps``, ``logit_scale`` and ``layers``, a list with one entry per layer: ``type`` (which mixer:
``rglru`` or ``parallel``), ``mixer`` (its sizes and constants) and ``mlp`` (``null``, dense or a mixture of experts).  Layers need not
be alike and come in any order.

* ``rglru``: ``width`` (channels of the recurrence), ``conv`` (taps of the short convolution), ``blocks`` (equal parts of the
  channels with gate matrices of their own).
* ``parallel``: ``left`` (chunked attention: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (positions per chunk),
  ``rot.dims``, ``rot.base``), ``right`` (gated linear attention: ``heads``, ``dim``, ``vdim``, ``tau``), ``left_scale``, ``right_scale``.
* ``mlp``: ``kind`` = ``dense`` with ``ff``, or ``moe`` with ``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top`` and optionally
  ``router.groups.count|keep`` and ``router.identity`` (router outputs behind the experts' that stand for the input itself).

Every size and constant is taken from the file; a missing required key, an unknown kind or sizes that contradict one another
raise ``ConfigError``.  Optional: ``mask`` and ``rot`` (absent: no chunks, no rotation), ``kv_heads`` (as many as ``heads``), ``vdim``
(like ``dim``), ``right.a_rank`` (the inner size of the low-rank decay projection, which only the random-weights writer needs: a
checkpoint's tensors fix it otherwise) and ``eos_token_id``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .givirax_config import _get
from .model_config import ConfigError


@dataclass(frozen=True)
class GatedLRUConfig:
    width: int
    conv: int
    blocks: int


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int = 0                # 0: all earlier positions
    rot_dims: int = 0             # 0: no rotation
    rot_base: float = 10000.0


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    a_rank: Optional[int] = None


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: ChunkedAttentionConfig
    right: GatedLinearConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class SumevikMlpConfig:
    kind: str                     # "dense" | "moe"
    ff: int
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1
    identity: int = 0


@dataclass(frozen=True)
class SumevikLayerConfig:
    type: str
    mixer: Union[GatedLRUConfig, ParallelMixerConfig]
    mlp: Optional[SumevikMlpConfig]


def _section(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"config.json: required key '{where}{key}' is missing")
    return v


def _chunked(m: Mapping[str, Any], w: str) -> ChunkedAttentionConfig:
    heads, dim = _get(m, "heads", int, w), _get(m, "dim", int, w)
    rot = m.get("rot")
    c = ChunkedAttentionConfig(
        heads=heads, kv_heads=_get(m, "kv_heads", int, w, heads, required=False), dim=dim,
        vdim=_get(m, "vdim", int, w, dim, required=False), scale=_get(m, "scale", float, w),
        chunk=_get(m.get("mask") or {}, "size", int, w + "mask.", 0, required=False),
        rot_dims=_get(rot, "dims", int, w + "rot.") if rot is not None else 0,
        rot_base=_get(rot, "base", float, w + "rot.") if rot is not None else 10000.0)
    if min(c.heads, c.kv_heads, c.dim, c.vdim) <= 0 or c.heads % c.kv_heads or c.chunk < 0:
        raise ConfigError(f"config.json: {w}: {c.heads} heads over {c.kv_heads} key heads, sizes {c.dim} and {c.vdim}, chunks of {c.chunk}")
    if c.rot_dims < 0 or c.rot_dims % 2 or c.rot_dims > c.dim or c.rot_base <= 0:
        raise ConfigError(f"config.json: {w}rot: {c.rot_dims} turned elements of {c.dim}, base {c.rot_base}")
    return c


def _linear(m: Mapping[str, Any], w: str) -> GatedLinearConfig:
    c = GatedLinearConfig(heads=_get(m, "heads", int, w), dim=_get(m, "dim", int, w), vdim=_get(m, "vdim", int, w),
                          tau=_get(m, "tau", float, w), a_rank=_get(m, "a_rank", int, w, None, required=False))
    if min(c.heads, c.dim, c.vdim) <= 0 or c.tau <= 0 or (c.a_rank is not None and c.a_rank <= 0):
        raise ConfigError(f"config.json: {w}: {c.heads} heads of {c.dim} x {c.vdim}, tau {c.tau}")
    return c


def _mlp(f: Mapping[str, Any], w: str) -> SumevikMlpConfig:
    kind = _get(f, "kind", str, w)
    if kind == "dense":
        c = SumevikMlpConfig("dense", _get(f, "ff", int, w))
        if c.ff <= 0:
            raise ConfigError(f"config.json: {w}ff must be positive")
        return c
    if kind != "moe":
        raise ConfigError(f"config.json: {w}kind '{kind}' is unknown; known: dense, moe")
    e, r = _section(f, "expert", w), _section(f, "router", w)
    g = r.get("groups") or {}
    c = SumevikMlpConfig("moe", _get(e, "ff", int, w + "expert."), limit=_get(e, "limit", float, w + "expert."),
                         experts=_get(r, "experts", int, w + "router."), top=_get(r, "top", int, w + "router."),
                         groups=_get(g, "count", int, w + "router.groups.", 1, required=bool(g)),
                         keep=_get(g, "keep", int, w + "router.groups.", 1, required=bool(g)),
                         identity=_get(r, "identity", int, w + "router.", 0, required=False))
    outputs = c.experts + c.identity
    if c.ff <= 0 or c.experts <= 0 or c.identity < 0 or c.limit <= 0:
        raise ConfigError(f"config.json: {w}: {c.experts} experts of inner size {c.ff} and limit {c.limit}, {c.identity} identity experts")
    if c.groups <= 0 or outputs % c.groups or not (0 < c.keep <= c.groups) or not (0 < c.top <= c.keep * (outputs // c.groups)):
        raise ConfigError(f"config.json: {w}router: top {c.top} of the best {c.keep} of {c.groups} groups over {outputs} outputs")
    return c


@dataclass(frozen=True)
class SumevikConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[SumevikLayerConfig, ...]
    eos_token_ids: tuple = ()
    architecture: str = "Sumevik"

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "SumevikConfig":
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        parsed = []
        for i, entry in enumerate(layers):
            where = f"layers[{i}]."
            kind = _get(entry, "type", str, where)
            m, w = _section(entry, "mixer", where), where + "mixer."
            if kind == "rglru":
                mixer = GatedLRUConfig(width=_get(m, "width", int, w), conv=_get(m, "conv", int, w), blocks=_get(m, "blocks", int, w))
                if min(mixer.width, mixer.conv, mixer.blocks) <= 0 or mixer.width % mixer.blocks:
                    raise ConfigError(f"config.json: {w}: {mixer.width} channels in {mixer.blocks} parts, {mixer.conv} taps")
            elif kind == "parallel":
                mixer = ParallelMixerConfig(left=_chunked(_section(m, "left", w), w + "left."), right=_linear(_section(m, "right", w), w + "right."),
                                            left_scale=_get(m, "left_scale", float, w), right_scale=_get(m, "right_scale", float, w))
            else:
                raise ConfigError(f"config.json: {where}type '{kind}' is not a mixer of this design; known: rglru, parallel")
            f = entry.get("mlp")
            parsed.append(SumevikLayerConfig(kind, mixer, _mlp(f, where + "mlp.") if f is not None else None))
        eos = d.get("eos_token_id")
        eos = tuple(int(x) for x in eos) if isinstance(eos, (list, tuple)) else ((int(eos),) if eos is not None else ())
        cfg = SumevikConfig(vocab=_get(d, "vocab", int, ""), width=_get(d, "width", int, ""),
                            norm_eps=_get(d.get("norm") or {}, "eps", float, "norm."),
                            logit_scale=_get(d, "logit_scale", float, "", 1.0, required=False), layers=tuple(parsed), eos_token_ids=eos)
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: vocab and width must be positive")
        return cfg
