"""The Sutuvik configuration reader, its model description, its tensor names, its caches and the plain
implementation's own small checks (no GPU)."""

import copy
import math

import pytest
import torch

import plain_sutuvik as plain
from cloud_inference_from_scratch_b200 import models, parts  # noqa: F401  (registries)
from cloud_inference_from_scratch_b200.config import ConfigError, resolve_config
from cloud_inference_from_scratch_b200.config.sutuvik_config import SutuvikConfig
from cloud_inference_from_scratch_b200.models import DecoderModel

F = torch.float64


def raw_config():
    rot = dict(base=3000.0, dims=6, scaling=dict(factor=4.0, low=1.5, high=6.0, original=100))
    biased = dict(heads=6, kv_heads=3, dim=8, vdim=10, scale=0.3, q_temp=dict(coef=0.2, every=9), v_mix=True)
    rotated = dict(heads=4, kv_heads=2, dim=12, vdim=15, scale=0.25, softcap=20.0, rot=rot, v_mix=True)
    mamba = dict(heads=6, vdim=5, state=7, groups=2, conv=4, norm_groups=3)
    moe = dict(kind="moe", expert=dict(ff=16), router=dict(experts=6, top=2, groups=dict(count=3, keep=2)))
    return dict(architecture="Sutuvik", vocab=50, width=24, logit_scale=0.7, norm=dict(eps=1e-5, groups=3),
                canon=dict(taps=4), token_side=dict(dim=5),
                layers=[dict(type="attention", mixer=dict(biased, v_mix=False), mlp=moe),
                        dict(type="attention_2", mixer=rotated, mlp=None),
                        dict(type="mamba2", mixer=mamba, mlp=moe),
                        dict(type="attention", mixer=biased, mlp=moe)])


def test_reads_back_what_it_wrote_and_is_found_by_its_name():
    raw = raw_config()
    arch, config, spec = resolve_config(raw)
    assert arch.name == "Sutuvik" and isinstance(config, SutuvikConfig)
    assert SutuvikConfig.from_dict(config.to_dict()) == config and config.to_dict() == raw
    assert spec.logit_scale == 0.7 and spec.head_tensor == "embed"
    assert [entry.layer for entry in spec.schedule] == [0, 1, 2, 3]


def test_the_first_layer_with_mixed_values_keeps_and_the_others_blend():
    model = DecoderModel(resolve_config(raw_config())[2])
    kinds = [getattr(layer.mixer.inner, "value_mix", None) for layer in model.layers]
    assert kinds == [None, "keep", None, "blend"]


def test_tensor_names_shapes_and_caches():
    model = DecoderModel(resolve_config(raw_config())[2])
    table = model.tensor_table()
    assert table["embed"].shape == (50, 24) and table["embed.norm"].shape == (24,) and table["final.norm"].shape == (24,)
    assert table["side.embed"].shape == (50, 20) and "head" not in table
    for index in range(4):
        assert table[f"l{index}.norm1"].shape == (24,) and table[f"l{index}.canon1"].shape == (24, 4)
        assert table[f"l{index}.side.gate"].shape == (5, 24) and table[f"l{index}.side.proj"].shape == (24, 5)
        assert table[f"l{index}.side.norm"].shape == (24,)
    assert table["l0.mix.q"].shape == (48, 24) and table["l0.mix.k"].shape == (24, 24) and table["l0.mix.v"].shape == (30, 24)
    assert table["l0.mix.q.norm"].shape == (8,) and table["l0.mix.k.norm"].shape == (8,) and table["l0.mix.sink"].shape == (6,)
    assert table["l0.mix.g"].shape == (6, 24) and table["l0.mix.o"].shape == (24, 60) and "l0.mix.vmix" not in table
    assert table["l1.mix.temp"].shape == (4,) and table["l1.mix.vmix"].shape == () and "l1.mix.sink" not in table
    assert "l1.mix.q.norm" not in table and "l1.mix.g" not in table and "l1.norm2" not in table
    assert not any(name.startswith("l1.mlp") for name in table)
    assert table["l2.mix.in"].shape == (2 * 30 + 2 * 14 + 6, 24) and table["l2.mix.conv"].shape == (58, 4)
    assert table["l2.mix.conv.b"].shape == (58,) and table["l2.mix.norm"].shape == (30,) and table["l2.mix.o"].shape == (24, 30)
    assert all(table[f"l2.mix.{name}"].shape == (6,) for name in ("dt_bias", "A_log", "D"))
    assert table["l2.mlp.router"].shape == (6, 24) and table["l2.mlp.correction"].shape == (6,)
    assert table["l2.mlp.e5.gate"].shape == (16, 24) and table["l2.mlp.e0.down"].shape == (24, 16)
    needs = model.cache_needs()
    assert (needs[0].pages.kv_heads, needs[0].pages.head_dim, needs[0].pages.value_size, needs[0].pages.window) == (3, 8, 10, 0)
    assert needs[0].state.shape == (3 * 24,)                     # the input convolution's last three rows
    assert needs[2].pages is None
    # heads' matrices and the short convolution's history (rounded to whole 16-byte pieces), then the input's
    assert needs[2].state.shape == (6 * 7 * 5 + 3 * 58 + 3 * 24,)


def test_one_tap_keeps_no_history():
    raw = raw_config()
    raw["canon"]["taps"] = 1
    needs = DecoderModel(resolve_config(raw)[2]).cache_needs()
    assert needs[0].state is None and needs[2].state.shape == (6 * 7 * 5 + 3 * 58,)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "positive"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "within a head"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(low=7.0), "low"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0), "positive"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=16), "v_mix"),
    (lambda c: c["layers"][2]["mixer"].update(groups=4), "multiple"),
    (lambda c: c["layers"][2]["mixer"].update(norm_groups=4), "divide"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=5), "choose from"),
    (lambda c: c["layers"][2]["mlp"]["router"]["groups"].update(count=4), "equal groups"),
    (lambda c: c["layers"][2]["mlp"].update(kind="dense"), "not built"),
    (lambda c: c["norm"].update(groups=5), "divide"),
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c.pop("token_side"), "token_side"),
])
def test_refusals(change, message):
    raw = copy.deepcopy(raw_config())
    change(raw)
    with pytest.raises(ConfigError, match=message):
        SutuvikConfig.from_dict(raw)


def test_plain_mechanisms_against_their_definitions():
    """The oracle's own pieces on inputs whose answer is known."""
    g = torch.Generator().manual_seed(1)
    x = torch.randn(3, 12, generator=g, dtype=F)
    y = plain.group_norm(x, torch.ones(12, dtype=F), 0.0, 4).view(3, 4, 3)
    assert torch.allclose((y * y).mean(-1), torch.ones(3, 4, dtype=F))
    # a filter that is one at the last tap copies; at the first of three it looks two tokens back
    w = torch.zeros(12, 3, dtype=F)
    w[:, 2] = 1.0
    assert torch.equal(plain.causal_conv(x, w), x)
    w[:, 2], w[:, 0] = 0.0, 1.0
    assert torch.equal(plain.causal_conv(x, w)[2], x[0]) and plain.causal_conv(x, w)[:2].abs().max() == 0
    # waves shorter than original / high stay, longer than original / low are divided
    rot = dict(base=1e4, dims=16, scaling=dict(factor=8.0, low=1.0, high=4.0, original=64))
    got, base = plain.wavelength_frequencies(rot), plain.wavelength_frequencies(dict(rot, scaling=None))
    ratio = got / base
    assert math.isclose(ratio[0], 1.0) and math.isclose(ratio[-1], 1 / 8)
    assert all(1 / 8 - 1e-9 <= r <= 1 + 1e-9 for r in ratio.tolist()) and ((ratio > 0.13) & (ratio < 0.99)).any()
    turned = plain.rotate_pairs(x.view(3, 1, 12), torch.arange(3), dict(base=100.0, dims=4))
    assert torch.equal(turned[..., 4:].reshape(3, 8), x[:, 4:]) and torch.allclose(turned.norm(dim=-1)[:, 0], x.norm(dim=-1))
    # the temperature steps up at the position whose count of tokens fills another `every`
    heat = plain.query_temperature(torch.arange(7), 0.5, 3)
    assert heat[0] == heat[1] == 1.0 and math.isclose(heat[2], 1 + 0.5 * math.log(2)) and math.isclose(heat[6], 1 + 0.5 * math.log(3))
    assert plain.head_slopes(8).tolist() == [2.0 ** -(h + 1) for h in range(8)]
    # a slope without scores: weights fall by exp(-slope) a token; a sink of -inf weight leaves them at sum one
    q, k, v = torch.zeros(4, 1, 2, dtype=F), torch.zeros(4, 1, 2, dtype=F), torch.eye(4, dtype=F).view(4, 1, 4)
    weights = plain.attend(q, k, v, 1.0, [-1e9], slopes=[0.5])[:, 0]
    assert torch.allclose(weights.sum(-1), torch.ones(4, dtype=F)) and math.isclose(weights[3, 3] / weights[3, 2], math.exp(0.5))
    # one in the denominator: a single key of score zero gets half the weight
    assert math.isclose(plain.attend(q, k, v, 1.0, [0.0])[0, 0, 0], 0.5)
    # a decay of one keeps everything; groups share B and C
    x, b, c = (torch.randn(5, 4, 3, generator=g, dtype=F), torch.randn(5, 2, 6, generator=g, dtype=F),
               torch.randn(5, 2, 6, generator=g, dtype=F))
    dt = torch.rand(5, 4, generator=g, dtype=F)
    y, _ = plain.state_space(x, b, c, dt, torch.full((4,), -1e3, dtype=F), torch.zeros(4, dtype=F))
    want = sum(dt[j, 3] * (c[4, 1] @ b[j, 1]) * x[j, 3] for j in range(5))
    assert torch.allclose(y[4, 3], want)
    # experts of a group that is not kept are never chosen, even with negative choice scores all round
    w = {"router": torch.zeros(6, 4, dtype=F), "correction": torch.tensor([-9.0, -9, -2, -3, -1, -9], dtype=F)}
    ids, share = plain.choose_experts(torch.ones(1, 4, dtype=F), w, dict(experts=6, top=2, groups=dict(count=3, keep=1)))
    assert sorted(ids[0].tolist()) == [2, 3] and torch.allclose(share, torch.full((1, 2), 0.5, dtype=F))
