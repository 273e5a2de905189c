"""Bozevik: from its typed configuration to a model description.

Token embedding; layers whose sublayers read the stream itself and whose results are layer-normalised (a gain, no bias)
before they join it; a mixer that is latent attention (queries through a normalised latent, interleaved rotary pairs on
a key part that all heads share), on its own cached latent or on an earlier layer's (``kv_from``), and that reads its
input moved towards the token before it; a clamped gated feed-forward that is dense or routed (sigmoid scores that
multiply the chosen experts' inputs, a shared expert beside them), or none; after every layer an average over the
embedding rows and everything the layers have left.  A final layer norm and the embedding table as head, its logits
times a constant.

Tensor names: ``embed``, ``final.norm``; per layer ``l<i>.`` + ``norm1``, ``norm2``, ``shift``, ``dwa``, ``mix.*``,
``mlp.*``.
"""

from __future__ import annotations

from ..config.bozevik_config import BozevikConfig, SharedLatentConfig, UnitConfig, UnitFeedForwardConfig
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 20     # the design names no limit; positions and angles are float32
SLOPE, UP_SHIFT = 1.702, 1.0     # g * sigmoid(SLOPE * g) * (u + UP_SHIFT)


def _mixer(config: BozevikConfig, mixer: SharedLatentConfig) -> PartSpec:
    position = PartSpec("rope_neox", dict(head_dim=mixer.rot_dim, rotary_dim=mixer.rot_dim, theta=mixer.base,
                                          max_positions=MAX_POSITIONS, pairing="interleaved", keep_pairing=True))
    inner = PartSpec("latent_attention",
                     dict(hidden_size=config.width, num_heads=mixer.heads, head_dim=mixer.dim, rot_dim=mixer.rot_dim,
                          value_dim=mixer.vdim, kv_rank=mixer.kv_rank, q_rank=mixer.q_rank, scale=mixer.scale,
                          position=position, norm_eps=config.norm_eps, shares_cache=mixer.kv_from is not None,
                          split_output=True),
                     prefix="mix.")
    return PartSpec("token_shift", dict(hidden_size=config.width, inner=inner, name="shift"))


def _unit(config: BozevikConfig, unit: UnitConfig, prefix: str) -> PartSpec:
    return PartSpec("clamped_glu", dict(hidden_size=config.width, intermediate_size=unit.ff, limit=unit.limit, slope=SLOPE,
                                        shift=UP_SHIFT, bias=False, split_output=True), prefix=prefix)


def _feed_forward(config: BozevikConfig, mlp: UnitFeedForwardConfig) -> PartSpec:
    if not mlp.experts:
        return _unit(config, mlp.unit, "mlp.")
    return PartSpec("routed_experts",
                    dict(hidden_size=config.width, intermediate_size=mlp.unit.ff, num_experts=mlp.experts, top=mlp.top,
                         correction=False, score="sigmoid", defer_sum=True, weight_inputs=True,
                         activation=(mlp.unit.limit, SLOPE, UP_SHIFT),
                         shared=_unit(config, mlp.shared, "shared.") if mlp.shared is not None else None),
                    prefix="mlp.")


def bozevik_spec(config: BozevikConfig) -> ModelSpec:
    norm = dict(hidden_size=config.width, eps=config.norm_eps, bias=False, names={"weight": ""})
    layers: list[LayerSpec] = []
    schedule: list[ScheduleEntry] = []
    for index, layer in enumerate(config.layers):
        parts = dict(mixer=_mixer(config, layer.mixer), mixer_norm=PartSpec("layernorm", norm, prefix="norm1"),
                     average=PartSpec("depth_average", dict(hidden_size=config.width, index=index,
                                                            states=len(config.layers) + 1, name="dwa"),
                                      family="connection"))
        if layer.mlp is not None:
            parts["feed_forward"] = _feed_forward(config, layer.mlp)
            parts["feed_forward_norm"] = PartSpec("layernorm", norm, prefix="norm2")
        layers.append(LayerSpec(prefix=f"l{index}.", block=PartSpec("postnorm_residual"), parts=parts))
        # layers and schedule entries run one to one, so a layer index is an entry index; the row before the first of
        # a step is every layer's own, whoever's latents it reads
        schedule.append(ScheduleEntry(layer=index, reads_cache_of=layer.mixer.kv_from,
                                      own_state=layer.mixer.kv_from is not None))
    return ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=config.width,
        embedding_tensor="embed",
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=PartSpec("layernorm", norm),
        final_norm_prefix="final.norm",
        head_tensor="embed",
        max_positions=MAX_POSITIONS,
        eos_token_id=None,
        logit_scale=config.logit_scale,
        # a layer without a feed-forward has no second norm to apply; a file may hold one all the same
        optional_tensors=tuple(f"l{i}.norm2" for i, layer in enumerate(config.layers) if layer.mlp is None),
    )


register_architecture("Bozevik", "bozevik", BozevikConfig.from_dict, bozevik_spec, replace=True)
