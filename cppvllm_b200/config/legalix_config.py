"""Typed configuration of the Legalix decoder, read from its ``config.json``.

Top level: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``residual_mult``, ``layers`` (a list with one entry per layer: ``type`` (which
mixer), ``mixer`` (its sizes and constants) and ``mlp`` (``null`` or dense)) and optionally ``loop``: layers ``start`` .. ``stop`` - 1 run ``times``
times in a row with the same weights.  Layers need not be alike and come in any order.

* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``softcap``, ``mask.size`` (positions in the window), ``mask.keep_first`` (first tokens
  that stay visible), ``rot.dims``, ``rot.base``.
* ``latent_attention``: ``heads``, ``dim`` (unturned), ``rot_dim`` (turned), ``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot.dims``, ``rot.base``.
* ``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv`` (taps), ``norm_groups``.
* ``mlp``: ``kind`` = ``dense`` with ``ff``.

Every size and constant is taken from the file; a missing required key, an unknown kind or sizes that contradict one another raise
``ConfigError``.  Optional: ``embedding.scale`` and ``residual_mult`` (1), ``loop``, ``mask`` (absent: all earlier positions), ``mask.keep_first`` (0),
``softcap`` (absent or null: none), ``rot`` (absent: no rotation), ``kv_heads`` (as many as ``heads``), ``vdim`` (like ``dim``), ``q_rank`` (absent: the
checkpoint's tensors fix it), ``groups`` and ``norm_groups`` (1) and ``eos_token_id``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .givirax_config import _get
from .model_config import ConfigError


@dataclass(frozen=True)
class WindowedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0          # 0: no cap
    window: int = 0               # 0: all earlier positions
    keep_first: int = 0
    rot_dims: int = 0             # 0: no rotation
    rot_base: float = 10000.0


@dataclass(frozen=True)
class SinkLatentAttentionConfig:
    heads: int
    dim: int                      # unturned query/key elements per head
    rot_dim: int                  # turned ones (the key's are shared by the heads)
    vdim: int
    q_rank: int                   # -1: whatever the checkpoint holds
    kv_rank: int
    scale: float
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class LegalixLayerConfig:
    type: str
    mixer: Union[WindowedAttentionConfig, SinkLatentAttentionConfig, StateSpaceConfig]
    ff: int = 0                   # 0: the layer has no feed-forward


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


def _attention(m: Mapping[str, Any], w: str) -> WindowedAttentionConfig:
    heads, dim = _get(m, "heads", int, w), _get(m, "dim", int, w)
    mask, rot = m.get("mask"), m.get("rot")
    cap = m.get("softcap")
    c = WindowedAttentionConfig(
        heads=heads, kv_heads=_get(m, "kv_heads", int, w, heads, required=False), dim=dim, vdim=_get(m, "vdim", int, w, dim, required=False),
        scale=_get(m, "scale", float, w), softcap=_get(m, "softcap", float, w) if cap is not None else 0.0,
        window=_get(mask, "size", int, w + "mask.") if mask is not None else 0,
        keep_first=_get(mask, "keep_first", int, w + "mask.", 0, required=False) if mask is not None else 0,
        rot_dims=_get(rot, "dims", int, w + "rot.") if rot is not None else 0,
        rot_base=_get(rot, "base", float, w + "rot.") if rot is not None else 10000.0)
    if min(c.heads, c.kv_heads, c.dim, c.vdim) <= 0 or c.heads % c.kv_heads:
        raise ConfigError(f"config.json: {w}: {c.heads} heads over {c.kv_heads} key heads, sizes {c.dim} and {c.vdim}")
    if (mask is not None and c.window <= 0) or c.keep_first < 0 or c.softcap < 0:
        raise ConfigError(f"config.json: {w}: a window of {c.window}, {c.keep_first} kept tokens, a cap of {c.softcap}")
    if c.rot_dims < 0 or c.rot_dims % 2 or c.rot_dims > c.dim or c.rot_base <= 0:
        raise ConfigError(f"config.json: {w}rot: {c.rot_dims} turned elements of {c.dim}, base {c.rot_base}")
    return c


def _latent(m: Mapping[str, Any], w: str) -> SinkLatentAttentionConfig:
    dim, rot_dim = _get(m, "dim", int, w), _get(m, "rot_dim", int, w)
    rot = m.get("rot")
    if not isinstance(rot, Mapping):
        raise ConfigError(f"config.json: required key '{w}rot' is missing")
    c = SinkLatentAttentionConfig(
        heads=_get(m, "heads", int, w), dim=dim, rot_dim=rot_dim, vdim=_get(m, "vdim", int, w, dim, required=False),
        q_rank=_get(m, "q_rank", int, w, -1, required=False), kv_rank=_get(m, "kv_rank", int, w), scale=_get(m, "scale", float, w),
        rot_dims=_get(rot, "dims", int, w + "rot.", rot_dim, required=False), rot_base=_get(rot, "base", float, w + "rot."))
    if min(c.heads, c.dim, c.rot_dim, c.vdim, c.kv_rank) <= 0 or c.q_rank == 0:
        raise ConfigError(f"config.json: {w}: sizes must be positive")
    if c.rot_dims <= 0 or c.rot_dims % 2 or c.rot_dims > c.rot_dim or c.rot_base <= 0:
        raise ConfigError(f"config.json: {w}rot: {c.rot_dims} turned elements (even, at most rot_dim = {c.rot_dim}), base {c.rot_base}")
    return c


def _state_space(m: Mapping[str, Any], w: str) -> StateSpaceConfig:
    c = StateSpaceConfig(heads=_get(m, "heads", int, w), vdim=_get(m, "vdim", int, w), state=_get(m, "state", int, w),
                         groups=_get(m, "groups", int, w, 1, required=False), conv=_get(m, "conv", int, w),
                         norm_groups=_get(m, "norm_groups", int, w, 1, required=False))
    if min(c.heads, c.vdim, c.state, c.groups, c.conv, c.norm_groups) <= 0 or c.heads % c.groups or (c.heads * c.vdim) % c.norm_groups:
        raise ConfigError(f"config.json: {w}: {c.heads} heads of {c.state} x {c.vdim} over {c.groups} groups, {c.conv} taps, {c.norm_groups} norm groups")
    return c


_MIXERS = {"attention": _attention, "latent_attention": _latent, "mamba2": _state_space}


@dataclass(frozen=True)
class LegalixConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    layers: Tuple[LegalixLayerConfig, ...]
    loop: Optional[LoopConfig] = None
    eos_token_ids: tuple = ()
    architecture: str = "Legalix"

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "LegalixConfig":
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        parsed = []
        for i, entry in enumerate(layers):
            where = f"layers[{i}]."
            kind = _get(entry, "type", str, where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type '{kind}' is not a mixer of this design; known: {', '.join(_MIXERS)}")
            m = entry.get("mixer")
            if not isinstance(m, Mapping):
                raise ConfigError(f"config.json: required key '{where}mixer' is missing")
            mixer = _MIXERS[kind](m, where + "mixer.")
            f, ff = entry.get("mlp"), 0
            if f is not None:
                fk = _get(f, "kind", str, where + "mlp.")
                if fk != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind '{fk}' is unknown; known: dense")
                ff = _get(f, "ff", int, where + "mlp.")
                if ff <= 0:
                    raise ConfigError(f"config.json: {where}mlp: inner size must be positive")
            parsed.append(LegalixLayerConfig(kind, mixer, ff))
        loop = d.get("loop")
        if loop is not None:
            loop = LoopConfig(_get(loop, "start", int, "loop."), _get(loop, "stop", int, "loop."), _get(loop, "times", int, "loop."))
            if not (0 <= loop.start < loop.stop <= len(parsed)) or loop.times <= 0:
                raise ConfigError(f"config.json: loop over layers {loop.start} .. {loop.stop} of {len(parsed)}, {loop.times} times")
        eos = d.get("eos_token_id")
        eos = tuple(int(x) for x in eos) if isinstance(eos, (list, tuple)) else ((int(eos),) if eos is not None else ())
        cfg = LegalixConfig(vocab=_get(d, "vocab", int, ""), width=_get(d, "width", int, ""),
                            norm_eps=_get(d.get("norm") or {}, "eps", float, "norm."),
                            embedding_scale=_get(d.get("embedding") or {}, "scale", float, "embedding.", 1.0, required=False),
                            residual_mult=_get(d, "residual_mult", float, "", 1.0, required=False), layers=tuple(parsed), loop=loop, eos_token_ids=eos)
        if cfg.vocab <= 0 or cfg.width <= 0:
            raise ConfigError("config.json: vocab and width must be positive")
        return cfg
