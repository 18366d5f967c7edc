"""Legalix as data: the typed configuration becomes a ``ModelSpec``.

A decoder-only model with a residual stream summed in 32-bit whose layers have ONE norm, read by the mixer and the feed-forward alike:
x <- x + m (mixer(n(x)) + ff(n(x))).  Mixer and feed-forward are members of one ``side_by_side`` group: their input projections are one product,
their output projections another, and the multiplier m rides on what lies between.  The norms are ``dynamic_tanh``.  Layers come in any order
with one of three mixers: grouped-query attention inside a window that keeps the first tokens, with capped scores (``masked_attention``), attention
over a cached latent with a sink (``latent_attention``) and a state-space recurrence (``ssd``).  A run of layers may be gone through several times;
in front of every pass the stream becomes a product of itself and the embedding output (``concat_input``), and every pass has its own cache
entries and state.  Tensor names: ``embed``, ``loop.in``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.legalix_config import LegalixConfig, SinkLatentAttentionConfig, WindowedAttentionConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def build_legalix_spec(cfg: LegalixConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    layers, positions = [], {}

    def rotation(dims: int, base: float, pairing: str) -> str:
        name = f"rot{dims}_{base!r}_{pairing}"
        positions.setdefault(name, PartSpec("rotary", dict(rotary_dim=dims, theta=base, max_positions=0, pairing=pairing)))
        return name

    def norm(prefix: str, name: str, **extra) -> PartSpec:
        return PartSpec("dynamic_tanh", dict(size=D, weight_name=name, **extra), prefix=prefix)

    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, WindowedAttentionConfig):
            params = dict(hidden_size=D, num_heads=m.heads, num_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, eps=eps, qk_norm=False,
                          window=m.window, keep_first=m.keep_first, softcap=m.softcap)
            if m.rot_dims:
                params["position"] = rotation(m.rot_dims, m.rot_base, "half")
            mixer = PartSpec("masked_attention", params, prefix=p + "mix.")
        elif isinstance(m, SinkLatentAttentionConfig):
            mixer = PartSpec("latent_attention", dict(
                hidden_size=D, num_heads=m.heads, nope_dim=m.dim, rot_dim=m.rot_dim, value_dim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank,
                scale=m.scale, eps=eps, position=rotation(m.rot_dims, m.rot_base, "interleaved"), rot=m.rot_dims, gate="none", sink=True),
                prefix=p + "mix.")
        else:
            mixer = PartSpec("ssd", dict(hidden_size=D, num_heads=m.heads, groups=m.groups, state=m.state, vdim=m.vdim, taps=m.conv,
                                         norm_parts=m.norm_groups, eps=eps), prefix=p + "mix.")
        members = [mixer]
        if layer.ff:
            members.append(PartSpec("gated_mlp", dict(hidden_size=D, intermediate_size=layer.ff, activation="gelu_tanh"), prefix=p + "mlp."))
        layers.append(LayerSpec(mixer=PartSpec("side_by_side", dict(hidden_size=D, scales=(cfg.residual_mult,) * len(members), members=tuple(members))),
                                ffn=None, mixer_norm=norm(p, "norm1"), block="parallel"))
    order, inputs = [RunEntry(i) for i in range(len(layers))], {}
    if cfg.loop is not None:
        a, b = cfg.loop.start, cfg.loop.stop
        inputs["loop"] = PartSpec("concat_input", dict(hidden_size=D, weight_name="in"), prefix="loop.")
        passes = [RunEntry(i, input="loop" if i == a else None, input_index=t) for t in range(cfg.loop.times) for i in range(a, b)]
        order = order[:a] + passes + order[b:]
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=D,
        vocab_size=cfg.vocab,
        embedding=PartSpec("scaled_positions", dict(vocab_size=cfg.vocab, hidden_size=D, scale=cfg.embedding_scale)),
        layers=layers,
        final_norm=norm("final.", "norm", buffer="head_normed"),
        lm_head=PartSpec("lm_head", dict(vocab_size=cfg.vocab, hidden_size=D), names={"weight": "head"}),
        positions=positions,
        run_order=order,
        inputs=inputs,
        eos_token_ids=tuple(cfg.eos_token_ids),
        residual_dtype="float32",
    )


register_architecture("Legalix", LegalixConfig.from_dict, build_legalix_spec, model_types=("legalix",), replace=True, builtin=True)
