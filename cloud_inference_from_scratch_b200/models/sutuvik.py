"""Sutuvik: from its typed configuration to a model description.

Token embedding whose rows pass a norm; pre-norm layers (RMS norm in groups of neighbouring elements) whose mixer reads
its normalised input plus a short causal convolution of it; a mixer that is a state-space recurrence (Mamba-2), softmax
attention without rotation (q and k normalised per head with gains, a query temperature that grows with the position, a
penalty proportional to the distance, a stored sink, one gate a head) or softmax attention with interleaved rotary
pairs (frequencies scaled by wavelength; q and k of unit size after the rotation, a stored factor per head and a soft
cap on the scores, one in the denominator); in both kinds of attention the values may be blended with those of the
first such layer; routed experts (sigmoid scores, a choice among the best groups of experts, weights of sum 1) or no
feed-forward; then a side input read from a table of the tokens.  A final norm and the embedding table as head, its
logits times a constant.

Tensor names: ``embed``, ``embed.norm``, ``side.embed``, ``final.norm``; per layer ``l<i>.`` + ``norm1``, ``norm2``,
``canon1``, ``mix.*``, ``mlp.*``, ``side.*``.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..config.sutuvik_config import BiasedAttentionConfig, Mamba2Config, RotatedAttentionConfig, SutuvikConfig

MAX_POSITIONS = 1 << 20     # the design names no limit; positions and angles are float32
WEIGHT_FLOOR = 1e-20        # joins the sum that the chosen experts' scores are divided by

ATTENTION_NAMES = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
                   "q_norm": "q.norm", "k_norm": "k.norm", "sink": "sink", "gate": "g", "factor": "temp",
                   "value_mix": "vmix"}


def _mixer(config: SutuvikConfig, mixer: Mamba2Config | BiasedAttentionConfig | RotatedAttentionConfig,
           value_mix: str | None) -> PartSpec:
    if isinstance(mixer, Mamba2Config):
        return PartSpec("mamba2", dict(hidden_size=config.width, num_heads=mixer.heads, value_dim=mixer.vdim,
                                       state_dim=mixer.state, num_groups=mixer.groups, taps=mixer.conv,
                                       norm_groups=mixer.norm_groups, eps=config.norm_eps), prefix="mix.")
    common = dict(hidden_size=config.width, num_heads=mixer.heads, num_kv_heads=mixer.kv_heads, head_dim=mixer.dim,
                  value_dim=mixer.vdim, qkv_bias=False, scale=mixer.scale, projection_float32=True,
                  norm_eps=config.norm_eps, names=ATTENTION_NAMES, value_mix=value_mix)
    if isinstance(mixer, BiasedAttentionConfig):
        return PartSpec("attention", dict(common, position=None, qk_norm="head", query_heat=mixer.heat, sink=True,
                                          distance_slopes=True, head_gate=True), prefix="mix.")
    rotation = PartSpec("rope_neox", dict(head_dim=mixer.dim, rotary_dim=mixer.rot.dims, theta=mixer.rot.base,
                                          max_positions=MAX_POSITIONS, pairing="interleaved", bands=mixer.rot.scaling,
                                          keep_pairing=True))
    return PartSpec("attention", dict(common, position=rotation, qk_norm="unit", head_factor=True, softcap=mixer.softcap,
                                      sink="one"), prefix="mix.")


def sutuvik_spec(config: SutuvikConfig) -> ModelSpec:
    norm = dict(hidden_size=config.width, eps=config.norm_eps, groups=config.norm_groups, name="")
    layers: list[LayerSpec] = []
    mixed = False
    for index, layer in enumerate(config.layers):
        value_mix = None
        if getattr(layer.mixer, "v_mix", False):
            value_mix, mixed = "blend" if mixed else "keep", True
        parts = dict(
            mixer_norm=PartSpec("group_rmsnorm", norm, prefix="norm1"),
            mixer=PartSpec("input_conv", dict(hidden_size=config.width, taps=config.canon_taps, name="canon1",
                                              inner=_mixer(config, layer.mixer, value_mix))),
            side=PartSpec("token_side", dict(hidden_size=config.width, dim=config.side_dim, index=index,
                                             layers=len(config.layers), vocab_size=config.vocab, eps=config.norm_eps,
                                             table="side.embed"), prefix="side.", family="feed_forward"))
        if layer.mlp is not None:
            parts["feed_forward_norm"] = PartSpec("group_rmsnorm", norm, prefix="norm2")
            parts["feed_forward"] = PartSpec(
                "routed_experts", dict(hidden_size=config.width, intermediate_size=layer.mlp.ff,
                                       num_experts=layer.mlp.experts, top=layer.mlp.top, correction=True,
                                       renormalize=True, score="sigmoid", groups=(layer.mlp.groups, layer.mlp.keep),
                                       norm_floor=WEIGHT_FLOOR, defer_sum=True), prefix="mlp.")
        layers.append(LayerSpec(prefix=f"l{index}.", block=PartSpec("prenorm_residual"), parts=parts))
    return ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=config.width,
        embedding_tensor="embed",
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(layer=i) for i in range(len(layers))),
        final_norm=PartSpec("group_rmsnorm", norm),
        final_norm_prefix="final.norm",
        head_tensor="embed",
        max_positions=MAX_POSITIONS,
        eos_token_id=None,
        logit_scale=config.logit_scale,
        embedding_norm=PartSpec("group_rmsnorm", norm),
        embedding_norm_prefix="embed.norm",
    )


register_architecture("Sutuvik", "sutuvik", SutuvikConfig.from_dict, sutuvik_spec, replace=True)
