"""The Bozevik configuration reader, its model description, its tensor names, its caches, the work lists of expanded
prompt attention and the plain implementation's own small checks (no GPU)."""

import copy
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_bozevik as plain
from cloud_inference_from_scratch_b200 import models, parts  # noqa: F401  (registries)
from cloud_inference_from_scratch_b200.cache.pools import CachePools, plan_groups
from cloud_inference_from_scratch_b200.config import ConfigError, resolve_config
from cloud_inference_from_scratch_b200.config.bozevik_config import BozevikConfig
from cloud_inference_from_scratch_b200.models import DecoderModel
from cloud_inference_from_scratch_b200.native.ops import LATENT_PROMPT_TOKENS, Ops

F = torch.float64


def raw_config():
    latent = dict(heads=3, dim=8, rot_dim=6, vdim=10, kv_rank=12, q_rank=20, scale=0.3, rot=dict(base=500.0, dims=6))
    moe = dict(kind="moe", expert=dict(ff=16, limit=0.7), router=dict(experts=5, top=2), shared=dict(ff=9, limit=1.2))
    return dict(architecture="Bozevik", vocab=50, width=24, norm=dict(eps=1e-5), logit_scale=0.7,
                layers=[dict(type="latent_attention", mixer=latent, mlp=dict(kind="dense", ff=40, limit=1.5)),
                        dict(type="latent_attention", mixer=dict(latent, kv_rank=8), mlp=None),
                        dict(type="latent_attention", mixer=dict(latent, heads=2, kv_from=0), mlp=moe),
                        dict(type="latent_attention", mixer=dict(latent, kv_rank=8, kv_from=1),
                             mlp={key: value for key, value in moe.items() if key != "shared"})])


def test_reads_back_what_it_wrote_and_is_found_by_its_name():
    raw = raw_config()
    arch, config, spec = resolve_config(raw)
    assert arch.name == "Bozevik" and isinstance(config, BozevikConfig)
    assert BozevikConfig.from_dict(config.to_dict()) == config and config.to_dict() == raw
    assert spec.logit_scale == 0.7 and spec.head_tensor == "embed"
    assert [(entry.layer, entry.reads_cache_of) for entry in spec.schedule] == [(0, None), (1, None), (2, 0), (3, 1)]
    assert [entry.own_state for entry in spec.schedule] == [False, False, True, True]


def test_tensor_names_and_shapes():
    model = DecoderModel(resolve_config(raw_config())[2])
    table = model.tensor_table()
    assert table["embed"].shape == (50, 24) and table["final.norm"].shape == (24,) and "head" not in table
    for index in range(4):
        assert table[f"l{index}.norm1"].shape == table[f"l{index}.shift"].shape == (24,)
        assert table[f"l{index}.dwa"].shape == (index + 2,)
        assert table[f"l{index}.mix.dq"].shape == (20, 24) and table[f"l{index}.mix.dq.norm"].shape == (20,)
    assert table["l0.mix.uq"].shape == (3 * 14, 20) and table["l2.mix.uq"].shape == (2 * 14, 20)
    assert table["l0.mix.dkv"].shape == (18, 24) and table["l1.mix.dkv"].shape == (14, 24)
    assert "l2.mix.dkv" not in table and "l2.mix.dkv.norm" not in table and table["l2.mix.uk"].shape == (16, 12)
    assert table["l3.mix.uv"].shape == (30, 8) and table["l0.mix.o"].shape == (24, 30)
    assert table["l0.mlp.gate"].shape == (40, 24) and not any(name.startswith("l1.mlp") for name in table)
    assert "l1.norm2" not in table and table["l0.norm2"].shape == (24,)
    assert table["l2.mlp.router"].shape == (5, 24) and table["l2.mlp.e4.down"].shape == (24, 16)
    assert table["l2.mlp.shared.up"].shape == (9, 24) and "l3.mlp.shared.up" not in table
    assert not any(name.endswith(".b") or "correction" in name for name in table)


def test_pages_are_shared_where_state_is_not():
    model = DecoderModel(resolve_config(raw_config())[2])
    needs = model.cache_needs()
    assert [need.owner for need in needs] == [0, 1, 0, 1]
    assert [need.state_owner for need in needs] == [0, 1, 2, 3]
    assert [need.pages.head_dim for need in needs] == [12, 8, 12, 8] and needs[0].pages.value_size == 6
    assert all(need.state.shape == (24,) and need.state.dtype == "float32" for need in needs)
    groups, place = plan_groups(needs, 2)
    assert len(groups) == 2 and sorted(place) == [0, 1]
    pools = CachePools(needs, groups, place, [7, 7], 4, 3, torch.float32, "cpu")
    bound = pools.bindings
    assert bound[2].kv.k.data_ptr() == bound[0].kv.k.data_ptr() and not bound[2].owns_cache
    assert len({binding.state.data_ptr() for binding in bound}) == 4 and all(b.state.shape == (3, 24) for b in bound)


def test_wrong_configurations_are_refused():
    def refused(change):
        raw = copy.deepcopy(raw_config())
        change(raw)
        with pytest.raises(ConfigError):
            resolve_config(raw)

    refused(lambda raw: raw["layers"][2]["mixer"].update(kv_from=2))              # itself
    refused(lambda raw: raw["layers"][3]["mixer"].update(kv_from=2))              # a layer that makes none
    refused(lambda raw: raw["layers"][2]["mixer"].update(kv_from=1))              # another latent size
    refused(lambda raw: raw["layers"][2]["mixer"].update(rot=dict(base=400.0, dims=6)))     # another rotation
    refused(lambda raw: raw["layers"][0]["mixer"]["rot"].update(dims=4))
    refused(lambda raw: raw["layers"][0]["mlp"].update(limit=0.0))
    refused(lambda raw: raw["layers"][0]["mlp"].update(kind="other"))
    refused(lambda raw: raw["layers"][2]["mlp"]["router"].update(top=6))
    refused(lambda raw: raw["layers"][0].update(type="attention"))
    refused(lambda raw: raw.pop("logit_scale"))
    refused(lambda raw: raw.update(layers=[]))


def test_a_second_norm_that_nothing_applies_may_be_in_the_file():
    assert resolve_config(raw_config())[2].optional_tensors == ("l1.norm2",)


@pytest.mark.parametrize("window", [0, 5, 300])
def test_work_lists_of_expanded_prompt_attention(window):
    """Every token of every portion lies in one tile, rows go on from request to request, and a portion's rows begin at
    the first key that any of its tokens sees."""
    lens, contexts = np.array([1, 1, 200, 2, 131]), np.array([9, 0, 40, 700, 0])
    host = SimpleNamespace(query_lens=lens, context_lens=contexts, num_single=2)
    plan = Ops.plan_latent_prompt(host, window)
    portions, blocks, tiles = plan["portions"], plan["block_portion"], plan["tiles"]
    assert portions[:-1, 0].tolist() == [2, 3, 4]
    first = [max(0, c + 1 - window) if window else 0 for c in contexts[2:]]
    assert portions[:-1, 2].tolist() == first
    rows = [int(c + n - f) for c, n, f in zip(contexts[2:], lens[2:], first)]
    assert portions[:, 1].tolist() == [0, rows[0], rows[0] + rows[1], sum(rows)]
    assert len(blocks) == -(-sum(rows) // 128)
    for b, p in enumerate(blocks):
        assert portions[p, 1] <= 128 * b < portions[p + 1, 1]
    covered = sorted((int(r), int(q0)) for r, q0, _, _ in tiles)
    assert covered == [(2, 0), (2, 128), (3, 0), (4, 0), (4, 128)]
    for r, q0, start, key in tiles:
        assert (start, key) == (portions[r - 2, 1], portions[r - 2, 2])
    seen = [contexts[r] - key + min(q0 + 128, lens[r]) for r, q0, _, key in tiles]
    assert seen == sorted(seen, reverse=True)
    few = SimpleNamespace(query_lens=np.array([1, LATENT_PROMPT_TOKENS - 1]), context_lens=np.array([5, 5]), num_single=1)
    assert Ops.plan_latent_prompt(few, window) == {}
    assert Ops.plan_latent_prompt(SimpleNamespace(query_lens=lens[:2], context_lens=contexts[:2], num_single=2), window) == {}
    many = SimpleNamespace(query_lens=np.array([64]), context_lens=np.array([1 << 18]), num_single=0)
    assert (Ops.plan_latent_prompt(many, window) == {}) == (window == 0)


# ------------------------------------------------------------------ the plain implementation's own checks
def test_the_plain_shift_and_average():
    x = torch.tensor([[1.0, 2.0], [5.0, 6.0], [0.0, 1.0]], dtype=F)
    share = torch.tensor([0.25, 1.0], dtype=F)
    assert plain.shifted(x, share).tolist() == [[0.75, 0.0], [4.0, 2.0], [1.25, 6.0]]
    assert plain.depth_average([x, 2 * x], torch.tensor([1.0, -0.5], dtype=F)).abs().max() == 0.0


def test_the_plain_unit_caps_one_side_of_the_gate_and_both_of_the_other():
    w = {"gate": torch.eye(1, dtype=F), "up": torch.eye(1, dtype=F), "down": torch.eye(1, dtype=F)}
    value = lambda z: float(plain.clamped_unit(torch.tensor([[z]], dtype=F), w, 2.0))  # noqa: E731
    sig = lambda z: 1 / (1 + np.exp(-z))  # noqa: E731
    assert value(5.0) == pytest.approx(2.0 * sig(1.702 * 2.0) * 3.0)
    assert value(-5.0) == pytest.approx(-5.0 * sig(-1.702 * 5.0) * -1.0)


def test_the_plain_router_scales_inputs():
    torch.manual_seed(0)
    w = {"router": torch.tensor([[1.0], [2.0]], dtype=F)}
    for e in range(2):
        for name in ("gate", "up", "down"):
            w[f"e{e}.{name}"] = torch.tensor([[0.5 + e]], dtype=F)
    h = torch.tensor([[0.8]], dtype=F)
    score = torch.sigmoid(2 * h)
    got = plain.routed_units(h, w, dict(router=dict(top=1), expert=dict(limit=9.0)))
    assert torch.allclose(got, plain.clamped_unit(score * h, plain.sub(w, "e1."), 9.0))
    assert not torch.allclose(got, score * plain.clamped_unit(h, plain.sub(w, "e1."), 9.0))


def test_the_plain_norm_takes_the_mean_off():
    x = torch.tensor([[3.0, 5.0]], dtype=F)
    assert torch.allclose(plain.centred_norm(x, torch.tensor([2.0, 1.0], dtype=F), 0.0), torch.tensor([[-2.0, 1.0]], dtype=F))
