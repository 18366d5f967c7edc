"""Sumevik as data: the typed configuration becomes a ``ModelSpec``.

A decoder-only model with a pre-norm residual stream summed in 32-bit whose norms store their weights around zero (1 + w is
used).  Layers come in any order with one of two mixers: a gated linear recurrence over channels behind a short convolution
(mixer ``gated_lru``), or two mixers side by side on the same input (mixer ``side_by_side``): grouped-query attention inside
chunks of positions with biases, normed and turned queries and keys and a gate per element (``masked_attention``), and linear
attention with a decay per key channel (``gated_linear``).  The feed-forward is absent, dense with a tanh-GELU gate
(``gated_mlp``), or a mixture of clamped gated experts (``routed_glu``) chosen inside the best groups by softmax scores with a
correction, some of whose outputs stand for the input itself.  The output head is the embedding table times a constant.
Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (``l<i>.mix.left.*|right.*``), ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sumevik_config import GatedLRUConfig, SumevikConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec


def build_sumevik_spec(cfg: SumevikConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    layers, positions = [], {}

    def norm(prefix: str, name: str, **extra) -> PartSpec:
        return PartSpec("rmsnorm_wide", dict(size=D, eps=eps, weight_name=name, offset=1.0, **extra), prefix=prefix)

    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, GatedLRUConfig):
            mixer = PartSpec("gated_lru", dict(hidden_size=D, width=m.width, taps=m.conv, blocks=m.blocks), prefix=p + "mix.")
        else:
            a, r = m.left, m.right
            left = dict(hidden_size=D, num_heads=a.heads, num_kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale, eps=eps,
                        chunk=a.chunk, qkv_bias=True, element_gate=True)
            if a.rot_dims:
                name = f"rot{a.rot_dims}_{a.rot_base!r}"
                positions.setdefault(name, PartSpec("rotary", dict(rotary_dim=a.rot_dims, theta=a.rot_base, max_positions=0, pairing="interleaved")))
                left["position"] = name
            right = dict(hidden_size=D, num_heads=r.heads, dim=r.dim, vdim=r.vdim, tau=r.tau, eps=eps, decay_rank=r.a_rank)
            mixer = PartSpec("side_by_side", dict(hidden_size=D, scales=(m.left_scale, m.right_scale), members=(
                PartSpec("masked_attention", left, prefix=p + "mix.left."), PartSpec("gated_linear", right, prefix=p + "mix.right."))))
        ffn = ffn_norm = None
        f = layer.mlp
        if f is not None:
            if f.kind == "dense":
                ffn = PartSpec("gated_mlp", dict(hidden_size=D, intermediate_size=f.ff, activation="gelu_tanh"), prefix=p + "mlp.")
            else:
                ffn = PartSpec("routed_glu", dict(hidden_size=D, intermediate_size=f.ff, num_experts=f.experts, top=f.top, score="softmax_all",
                                                  activation="clamped", limit=f.limit, router_bias=False, correction=True, groups=f.groups,
                                                  keep_groups=f.keep, identity=f.identity), prefix=p + "mlp.")
            ffn_norm = norm(p, "norm2")
        layers.append(LayerSpec(mixer=mixer, ffn=ffn, mixer_norm=norm(p, "norm1"), ffn_norm=ffn_norm, block="prenorm"))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=D,
        vocab_size=cfg.vocab,
        embedding=PartSpec("scaled_positions", dict(vocab_size=cfg.vocab, hidden_size=D)),
        layers=layers,
        # the constant in front of the logits rides on the final norm's weight: the rows the head reads are scaled in float
        final_norm=norm("final.", "norm", buffer="head_normed", gain=cfg.logit_scale),
        lm_head=PartSpec("lm_head", dict(vocab_size=cfg.vocab, hidden_size=D), names={"weight": "embed"}),
        positions=positions,
        eos_token_ids=tuple(cfg.eos_token_ids),
        residual_dtype="float32",
    )


register_architecture("Sumevik", SumevikConfig.from_dict, build_sumevik_spec, model_types=("sumevik",), replace=True, builtin=True)
