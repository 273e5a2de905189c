"""The Bozevik design in the engine against the plain implementation of ``plain_bozevik.py``: each mechanism alone,
whole prompts against decoding, portions down to two tokens, unequal batches, pages and state slots that are used
again, far keys and page edges, first tokens, long decoding, sizes of every kind, and greedy generation through the
public entry point."""

import copy
import json
import subprocess
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_bozevik as plain
from helpers import peak_tokens, random_tokens, replay, requests_in, trace_mixed, trace_portions, trace_tail, trace_whole

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
F = torch.float64

# worst |logit difference| of a row over the standard deviation of the request's reference logits
GATE = {"float32": 2e-4, "bfloat16": 0.1}


# ------------------------------------------------------------------ configurations
def latent(heads=3, dim=8, rot_dim=6, vdim=12, kv_rank=20, q_rank=28, scale=0.3, base=300.0, source=None):
    mixer = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale,
                 rot=dict(base=base, dims=rot_dim))
    if source is not None:
        mixer["kv_from"] = source
    return dict(type="latent_attention", mixer=mixer)


def dense(layer, ff=40, limit=1.5):
    return dict(layer, mlp=dict(kind="dense", ff=ff, limit=limit))


def moe(layer, ff=16, experts=5, top=2, limit=1.0, shared=(24, 2.0)):
    mlp = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    if shared:
        mlp["shared"] = dict(ff=shared[0], limit=shared[1])
    return dict(layer, mlp=mlp)


def bare(layer):
    return dict(layer, mlp=None)


def config(layers, width=64, vocab=211, eps=1e-5, scale=0.7):
    return dict(architecture="Bozevik", vocab=vocab, width=width, logit_scale=scale, norm=dict(eps=eps), layers=list(layers))


CONFIGS = {
    # two latents, each read by later layers with other head counts and sizes, every kind of feed-forward and none
    "mixed": config([dense(latent()), moe(latent(heads=2, dim=12, vdim=7, q_rank=9, source=0)),
                     bare(latent(kv_rank=24, rot_dim=8, base=1000.0)), moe(latent(source=0), top=1, shared=None),
                     dense(latent(heads=5, kv_rank=24, rot_dim=8, base=1000.0, source=2), limit=0.6)]),
    # one layer, one head, everything that can be one is one; latent and key part of equal size
    "plain": config([moe(latent(heads=1, dim=16, rot_dim=16, vdim=16, kv_rank=16, q_rank=16), ff=16, experts=1, top=1)],
                    width=48, vocab=130, scale=1.0),
    # sizes that are no multiples of eight or four, all experts chosen, a layer of attention alone first
    "narrow": config([bare(latent(heads=3, dim=5, rot_dim=2, vdim=3, kv_rank=9, q_rank=7)),
                      moe(latent(heads=2, dim=6, rot_dim=10, vdim=9, kv_rank=18, q_rank=5), ff=10, experts=3, top=3,
                          shared=(6, 0.5)),
                      dense(latent(heads=4, dim=3, rot_dim=2, vdim=5, kv_rank=9, q_rank=11, source=0), ff=7)],
                     width=37, vocab=77, eps=1e-6),
    # sizes that the tensor-core kernels take: twenty heads (more than one row tile), heads of 64 + 32 and of 40 + 16,
    # values of 64, 24 and 72, a latent of 64 and one of 200
    "tiles": config([dense(latent(heads=20, dim=64, rot_dim=32, vdim=64, kv_rank=64, q_rank=48, scale=0.12), ff=64),
                     moe(latent(heads=4, dim=40, rot_dim=32, vdim=24, kv_rank=64, q_rank=32, scale=0.2, source=0,), ff=32,
                         experts=8, top=3, shared=(48, 1.0)),
                     moe(latent(heads=3, dim=72, rot_dim=16, vdim=72, kv_rank=200, q_rank=64, scale=0.15), ff=48,
                         experts=4, top=2, shared=None)], width=128),
}
PAGE = {"mixed": 4, "plain": 16, "narrow": 8, "tiles": 16}
# N(0, 0.05) weights leave shifts, averages and scores close to nothing
SCALES = {"embed": 10.0, "shift": 8.0, "mix.dq": 2.0, "mix.uq": 4.0, "mix.uk": 4.0, "mix.uv": 2.0, "mix.dkv": 2.0,
          "dq.norm": 0.5, "dkv.norm": 0.5, "mlp.router": 8.0, "mlp.gate": 4.0, "mlp.up": 4.0, "mlp.e": 3.0, "shared": 1.5}
# ... and in the bfloat16 runs scores that differ less, so that rounding a query does not decide what a token reads
SCALES_BF16 = dict(SCALES, **{"mix.uq": 2.0, "mix.uk": 2.0})


def make_model(folder, raw, seed, std=0.05, scales=None):
    from cloud_inference_from_scratch_b200.weights import write_random_model

    return write_random_model(folder, raw, seed, std=std, scales=scales or SCALES)


def all_chosen(raw):
    """The same configuration with every expert chosen: nothing hangs on a choice that bfloat16 rounding decides."""
    raw = copy.deepcopy(raw)
    for layer in raw["layers"]:
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return raw


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("bozevik")
    out = {}
    for index, (name, raw) in enumerate(CONFIGS.items()):
        out[name, "float32"] = make_model(root / name, raw, 5 + index)
        out[name, "bfloat16"] = make_model(root / (name + "-all"), all_chosen(raw), 5 + index, scales=SCALES_BF16)
    return out


def core_for(folder, dtype, page, pages, slots=4, step_tokens=0):
    from cloud_inference_from_scratch_b200.engine.core import build_core

    return build_core(folder, dtype=dtype, page_size=page, num_pages=pages, max_requests=slots,
                      max_model_len=pages * page, max_tokens_per_step=step_tokens)


PLAIN_LOGITS = {}


def plain_logits(folder, tokens):
    key = (str(folder), tuple(tokens))
    if key not in PLAIN_LOGITS:
        raw, tensors = plain.read_folder(folder)
        PLAIN_LOGITS[key] = plain.forward(raw, tensors, tokens).numpy()
    return PLAIN_LOGITS[key]


def check(folder, got, dtype, gate=None):
    """Every row against the plain model run on the whole request."""
    limit = gate or GATE[dtype]
    worst = 0.0
    for rid, tokens in got["fed"].items():
        ref = plain_logits(folder, tokens)
        rows = got["logits"][rid]
        assert sorted(rows) == list(range(len(tokens))), f"{rid}: positions missing"
        mine = np.stack([rows[p] for p in range(len(tokens))])
        errors = np.abs(mine - ref).max(axis=1) / ref.std()
        worst = max(worst, float(errors.max()))
        assert errors.max() <= limit, (
            f"{rid}: first wrong position {int(np.argmax(errors > limit))} of {len(tokens)}, error {errors.max():.3e}")
    return worst


def run_trace(core, steps):
    return {"logits": replay(core, steps), "fed": requests_in(steps)}


def requests_for(raw, lengths, seed):
    return {f"r{i}": random_tokens(raw["vocab"], n, seed + i) for i, n in enumerate(lengths)}


# ------------------------------------------------------------------ the whole model, every cutting
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_decoding_portions_and_batches(folders, name, dtype):
    page, folder = PAGE[name], folders[name, dtype]
    # lengths: one token, two, a page's edge and one past it, several pages, more than a tile of 128 rows
    requests = requests_for(CONFIGS[name], [1, 2, page, page + 1, 61, 150], seed=10)
    for steps in (trace_whole(requests), trace_tail(requests, tail=40), trace_portions(requests),
                  trace_mixed(requests, seed=3, live_limit=3)):
        # a pool that holds what is live and no more, and three slots: pages and slots come back
        pages = -(-peak_tokens(steps, round_to=page) // page) + 1
        core = core_for(folder, dtype, page, pages, slots=3)
        check(folder, run_trace(core, steps), dtype)
        assert core.cache.free_pages(0) == core.cache.total_pages(0)


def test_long_portions_beside_single_tokens_and_short_ones(folders):
    """Steps in which single tokens, portions of two tokens and portions of more than a tile meet, over contexts of their
    own: every form of the attention in one step."""
    raw, folder = CONFIGS["tiles"], folders["tiles", "bfloat16"]
    tokens = requests_for(raw, [40, 300, 260, 180], seed=30)
    cuts = {"r0": [37, 1, 1, 1], "r1": [130, 2, 168], "r2": [3, 190, 66, 1], "r3": [1, 49, 130]}
    steps, place = [], {rid: 0 for rid in tokens}
    for index in range(4):
        entries, end = [], []
        for rid, sizes in cuts.items():
            if index < len(sizes):
                at = place[rid]
                place[rid] = at + sizes[index]
                entries.append(dict(id=rid, tokens=tokens[rid][at:place[rid]], want=list(range(sizes[index]))))
                if place[rid] == len(tokens[rid]):
                    end.append(rid)
        steps.append(dict(step=index, entries=entries, end=end))
    core = core_for(folder, "bfloat16", 16, 64)
    check(folder, run_trace(core, steps), "bfloat16")


def drawn_configuration(seed):
    """A configuration drawn from the whole space of sizes: widths, head counts, plain, rotated and value sizes (multiples
    of 8 and 16 and others, within and beyond what the tensor-core kernels take), latents from a few elements to more
    than the tensor-core decode kernel takes, layers that read any earlier latent, experts from one to many with one to
    all chosen, shared experts or none, layers without feed-forward."""
    import random

    rng = random.Random(seed)
    layers, owners = [], []
    for index in range(rng.randint(1, 6)):
        sizes = dict(heads=rng.choice([1, 2, 3, 5, 8, 16, 20]), dim=rng.choice([4, 8, 12, 32, 48, 64, 128]),
                     rot_dim=rng.choice([2, 8, 16, 32, 64]), vdim=rng.choice([3, 8, 16, 40, 64, 96, 128, 136]),
                     kv_rank=rng.choice([7, 8, 24, 64, 96, 256, 520]), q_rank=rng.choice([5, 16, 33, 64, 96]),
                     base=rng.choice([100.0, 10000.0, 500000.0]))
        if owners and rng.random() < 0.5:
            source = rng.choice(owners)
            sizes.update({key: layers[source]["mixer"][key] for key in ("kv_rank", "rot_dim")},
                         base=layers[source]["mixer"]["rot"]["base"], source=source)
        else:
            owners.append(index)
        sizes["scale"] = rng.choice([0.4, 1.0, 2.0]) / (sizes["dim"] + sizes["rot_dim"]) ** 0.5
        layer = latent(**sizes)
        kind = rng.choice(["none", "dense", "moe", "moe"])
        if kind == "dense":
            layer = dense(layer, rng.choice([8, 24, 100]), rng.choice([0.5, 1.5, 7.0]))
        elif kind == "moe":
            experts = rng.choice([1, 2, 4, 8, 13])
            layer = moe(layer, rng.choice([8, 10, 16, 48]), experts, rng.randint(1, min(experts, 4)), rng.choice([0.5, 2.0]),
                        rng.choice([None, (8, 1.0), (56, 3.0)]))
        else:
            layer = bare(layer)
        layers.append(layer)
    return config(layers, width=rng.choice([40, 64, 96, 130, 256]), vocab=rng.choice([50, 211, 450]),
                  eps=rng.choice([1e-6, 1e-5]), scale=rng.choice([0.25, 1.0]))


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_drawn_configurations(seed, tmp_path):
    raw = drawn_configuration(seed)
    requests = requests_for(raw, [1, 2, 37, 150], seed=seed)
    for dtype, scales, gate in (("float32", SCALES, 4e-4), ("bfloat16", SCALES_BF16, 0.2)):
        folder = make_model(tmp_path / dtype, raw if dtype == "float32" else all_chosen(raw), 100 + seed, scales=scales)
        for steps in (trace_whole(requests), trace_mixed(requests, seed=seed, live_limit=3)):
            pages = -(-peak_tokens(steps, round_to=16) // 16) + 1
            core = core_for(folder, dtype, 16, pages, slots=3)
            check(folder, run_trace(core, steps), dtype, gate=gate)


def test_float32_rows_do_not_depend_on_the_cut_or_the_batch(folders):
    """The same position through four cuttings: equal to rounding of the order of additions at most."""
    raw = CONFIGS["mixed"]
    requests = requests_for(raw, [50, 31, 77], seed=40)
    seen = []
    for steps in (trace_whole(requests), trace_tail(requests, tail=20), trace_portions(requests),
                  trace_mixed(requests, seed=9, live_limit=3)):
        core = core_for(folders["mixed", "float32"], "float32", 4, 64, slots=3)
        seen.append(replay(core, steps))
    for rid, tokens in requests.items():
        base = np.stack([seen[0][rid][p] for p in range(len(tokens))])
        for other in seen[1:]:
            mine = np.stack([other[rid][p] for p in range(len(tokens))])
            assert np.abs(mine - base).max() <= 5e-5 * base.std()


def test_long_decoding_over_many_pages(folders):
    for name in ("mixed", "tiles"):
        requests = requests_for(CONFIGS[name], [170, 165], seed=70)
        steps = trace_tail(requests, tail=160)
        for dtype in ("float32", "bfloat16"):
            core = core_for(folders[name, dtype], dtype, PAGE[name], 400 // PAGE[name], slots=2)
            check(folders[name, dtype], run_trace(core, steps), dtype)


def test_a_state_slot_that_is_used_again_starts_from_zero(folders):
    """One slot only: every request inherits the slot of the one before it, and its first row must see zeros there."""
    for name in ("plain", "mixed"):
        requests = requests_for(CONFIGS[name], [30, 1, 8, 19], seed=90)
        core = core_for(folders[name, "float32"], "float32", 16, 4, slots=1)
        check(folders[name, "float32"], run_trace(core, trace_portions(requests)), "float32")


def test_streams_after_every_layer(folders):
    folder = folders["mixed", "float32"]
    raw, tensors = plain.read_folder(folder)
    tokens = random_tokens(raw["vocab"], 33, 8)
    streams = []
    plain.forward(raw, tensors, tokens, streams)
    core = core_for(folder, "float32", 4, 16)
    got = []

    def look(index, residual, pending):
        rows = torch.arange(residual.shape[0], dtype=torch.int32).cuda()
        out = torch.empty_like(residual)
        core.runtime.ops.advance(residual, pending, out, rows=rows)
        got.append(out.cpu())

    core.model.after_layer = look
    from cloud_inference_from_scratch_b200.engine.step import StepEntry

    core.step.admit("a")
    core.step.run([StepEntry("a", tokens)])
    assert len(got) == len(streams)
    for mine, want in zip(got, streams):
        close(mine, want, "float32")


# ------------------------------------------------------------------ mechanisms alone
def runtime(dtype):
    from cloud_inference_from_scratch_b200.engine.runtime import Runtime

    return Runtime("cuda:0", dtype)


def rand(*shape, scale=1.0, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, dtype, scale=None, loose=3e-2, tight=2e-5):
    want = want.double().cpu()
    error = float((got.double().cpu() - want).abs().max() / (scale or want.std()))
    assert error <= (tight if dtype == "float32" else loose), error


def step_of(lengths, slots=None, active=None):
    singles = 0
    while singles < len(lengths) and lengths[singles] == 1:
        singles += 1
    starts = np.concatenate([[0], np.cumsum(lengths)]).astype(np.int32)
    request_of = np.repeat(np.arange(len(lengths)), lengths).astype(np.int32)
    put = lambda values: torch.tensor(np.asarray(values), dtype=torch.int32).cuda()  # noqa: E731
    return SimpleNamespace(num_requests=len(lengths), num_single=singles, query_start=put(starts),
                           request_of_token=put(request_of), slots=put(slots if slots is not None else range(len(lengths))),
                           request_active=put(active if active is not None else [1] * len(lengths)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [37, 64, 2048, 3001, 9000])
def test_normalised_updates_and_the_average_over_depth(dtype, width):
    """A mean far from zero beside a small spread; terms in every form an update may have; kept states, the average over
    them, all rows and chosen ones; the final norm of the result."""
    from cloud_inference_from_scratch_b200.lazy import DepthUpdate, NormedUpdate, Partials, WeightedTerms

    rt = runtime(dtype)
    rows, states, eps = 5, 4, 1e-5
    stream, history = rand(rows, width, seed=1), rand(rows, states * width, seed=2)
    gain, out_gain = 1 + rand(width, scale=0.2, seed=3), 1 + rand(width, scale=0.2, seed=4)
    share = rand(3, seed=5)
    first, second, third = rand(rows, width, scale=0.1, seed=6) + 7.0, rand(rows, width, seed=7), rand(rows, width, seed=8)
    weights = rand(rows, 2, seed=9)
    side = torch.stack([first, second], 1).reshape(rows, 2 * width).cuda().contiguous()
    both = torch.stack([first, second]).cuda().contiguous()
    forms = [(first.cuda(), first), (Partials(both, 2, rows, width, None), first + second),
             (WeightedTerms(side, weights.cuda()), weights[:, :1] * first + weights[:, 1:] * second),
             (WeightedTerms(side, None, count=2, extra=third.cuda()), first + second + third)]
    chosen = torch.tensor([4, 0, 4], dtype=torch.int32).cuda()
    for update, y in forms:
        y = y.double()
        for kind, added in (("plain", y), ("rms", plain.rms_norm(y, gain.double(), eps)),
                            ("centred", plain.centred_norm(y, gain.double(), eps))):
            pending = update if kind == "plain" else NormedUpdate(update, gain.cuda(), eps, centred=kind == "centred")
            # no history: the stream takes the update, and its rows come out rounded
            residual, out = stream.clone().cuda(), torch.empty(rows, width, dtype=rt.dtype).cuda()
            rt.ops.advance(residual, pending, out)
            row = stream.double() + added
            close(residual, row, "float32", scale=1.0, tight=1e-4)
            close(out, row, dtype, scale=float(row.abs().max()), loose=5e-3, tight=1e-5)
            # the row begins from a kept state and is kept there; the stream becomes the average
            held = history.clone().cuda()
            base = held[:, 2 * width:3 * width]
            residual = stream.clone().cuda()
            rt.ops.advance(residual, DepthUpdate(pending, base, held, 2, share.cuda()), out)
            parts = [history[:, j * width:(j + 1) * width].double() for j in range(3)]
            row = parts[2] + added
            mixed = plain.depth_average([parts[0], parts[1], row], share.double())
            close(held[:, 2 * width:3 * width], row, "float32", scale=1.0, tight=1e-4)
            assert torch.equal(held[:, :2 * width].cpu(), history[:, :2 * width])
            assert torch.equal(held[:, 3 * width:].cpu(), history[:, 3 * width:])
            close(residual, mixed, "float32", scale=1.0, tight=1e-4)
            close(out, mixed, dtype, scale=float(mixed.abs().max()), loose=5e-3, tight=1e-5)
            # chosen rows of the norm: nothing else is written
            held, residual = history.clone().cuda(), stream.clone().cuda()
            picked = torch.empty(3, width, dtype=rt.dtype).cuda()
            rt.ops.advance(residual, DepthUpdate(pending, held[:, 2 * width:3 * width], held, 2, share.cuda()), picked,
                           rows=chosen, norm=(out_gain.cuda(), eps))
            assert torch.equal(residual.cpu(), stream) and torch.equal(held.cpu(), history)
            want = plain.centred_norm(mixed, out_gain.double(), eps)[[4, 0, 4]]
            close(picked, want, dtype, scale=1.0, tight=2e-4)
    # midway: kept, but the stream stays; the first layer: the stream itself is kept
    held, residual = history.clone().cuda(), stream.clone().cuda()
    rt.ops.advance(residual, DepthUpdate(first.cuda(), None, held, 1, None), out, write=False)
    assert torch.equal(residual.cpu(), stream)
    close(held[:, width:2 * width], stream.double() + first.double(), "float32", scale=1.0, tight=1e-5)
    rt.ops.advance(residual, DepthUpdate(None, None, held, 0, None), out)
    assert torch.equal(held[:, :width].cpu(), stream) and torch.equal(residual.cpu(), stream)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [35, 64, 2056, 5000])
@pytest.mark.parametrize("pending", [True, False])
def test_the_shift_reads_the_row_before_and_leaves_the_last(dtype, width, pending):
    """Requests of one token, of two, of a run's length and more, one that is not active (its state must stay), slots in
    another order than the requests; states that are not zero; then the next step of the same requests."""
    from cloud_inference_from_scratch_b200.lazy import NormedUpdate

    rt = runtime(dtype)
    rt.ops.require_stream_step()
    eps = 1e-5
    slots, lengths = [3, 0, 5, 1, 2], [1, 1, 2, 8, 21]
    share, gain = rand(width, scale=0.6, seed=1), 1 + rand(width, scale=0.2, seed=2)
    # the state lies behind another part of a wider slot
    wide = rand(6, 8 + (width + 3) // 4 * 4, seed=3).cuda()
    state, held = wide[:, 8:], wide.clone().double().cpu()
    for step, active in ((lengths, [1, 0, 1, 1, 1]), ([1] * 5, [1, 1, 1, 0, 1]), ([1, 7, 9, 16, 17], [1] * 5)):
        tokens = sum(step)
        ctx = step_of(step, slots, active)
        stream, y = rand(tokens, width, seed=tokens), rand(tokens, width, seed=tokens + 1)
        x = stream.double() + (plain.centred_norm(y.double(), gain.double(), eps) if pending else 0.0)
        residual, out = stream.clone().cuda(), torch.empty(tokens, width, dtype=rt.dtype).cuda()
        rt.ops.advance(residual, NormedUpdate(y.cuda(), gain.cuda(), eps, centred=True) if pending else None, out,
                       shift=(share.cuda(), state), ctx=ctx)
        rt.ops.check_errors()
        at = 0
        for request, count in enumerate(step):
            mine = held[slots[request], 8:8 + width]
            before = torch.cat([mine.unsqueeze(0), x[at:at + count - 1]])
            rows = x[at:at + count]
            want = rows + (before - rows) * share.double()
            close(out[at:at + count], want, dtype, scale=float(want.abs().max()), loose=5e-3, tight=1e-5)
            if active[request]:
                held[slots[request], 8:8 + width] = rows[-1]
            at += count
        close(residual, x, "float32", scale=1.0, tight=1e-4)
        close(wide, held, "float32", scale=1.0, tight=1e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,top,hidden,ff,shared", [(5, 2, 48, 16, 24), (1, 1, 40, 24, 0), (8, 8, 64, 32, 16),
                                                          (13, 3, 36, 10, 7), (6, 1, 256, 144, 40), (4, 2, 72, 8, 0)])
def test_routed_experts_with_weighted_inputs_a_clamp_and_a_shared_expert(dtype, experts, top, hidden, ff, shared):
    """The part alone, on inputs large enough that every bound is met: a weight on the output instead of the input, or a
    clamp left out, would show."""
    from cloud_inference_from_scratch_b200.config import PartSpec
    from cloud_inference_from_scratch_b200.parts import build_part

    rt = runtime(dtype)
    side = PartSpec("clamped_glu", dict(hidden_size=hidden, intermediate_size=shared, limit=0.9, bias=False), prefix="shared.")
    part = build_part("feed_forward", PartSpec("routed_experts", dict(
        hidden_size=hidden, intermediate_size=ff, num_experts=experts, top=top, correction=False, score="sigmoid",
        defer_sum=True, weight_inputs=True, activation=(0.7, 1.702, 1.0), shared=side if shared else None)))
    tensors = {"router": rand(experts, hidden, scale=0.3, seed=1)}
    for index, prefix in enumerate([f"e{e}." for e in range(experts)] + (["shared."] if shared else [])):
        inner = shared if prefix == "shared." else ff
        tensors[prefix + "gate"] = rand(inner, hidden, scale=0.3, seed=10 + index).to(rt.dtype)
        tensors[prefix + "up"] = rand(inner, hidden, scale=0.3, seed=40 + index).to(rt.dtype)
        tensors[prefix + "down"] = rand(hidden, inner, scale=0.3, seed=70 + index).to(rt.dtype)
    assert set(part.tensor_specs()) == set(tensors)
    part.bind({name: t.cuda() for name, t in tensors.items()}, rt)
    x = rand(150, hidden, seed=5).to(rt.dtype)
    for count in (150, 3):
        got = part.forward(x[:count].cuda(), SimpleNamespace())
        out = torch.empty(count, hidden, dtype=torch.float32).cuda()
        rt.ops.advance(torch.zeros(count, hidden).cuda(), got, out)
        rt.ops.check_errors()
        mlp = dict(router=dict(top=top), expert=dict(limit=0.7))
        if shared:
            mlp["shared"] = dict(limit=0.9)
        want = plain.routed_units(x[:count].double(), {name: t.double() for name, t in tensors.items()}, mlp)
        close(out, want, dtype, loose=4e-2, tight=2e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_are_told_apart_where_their_scores_round_to_one(dtype):
    from cloud_inference_from_scratch_b200.config import PartSpec
    from cloud_inference_from_scratch_b200.parts import build_part

    rt = runtime(dtype)
    part = build_part("feed_forward", PartSpec("routed_experts", dict(
        hidden_size=16, intermediate_size=16, num_experts=4, top=1, correction=False, score="sigmoid", defer_sum=True,
        weight_inputs=True, activation=(9.0, 1.702, 1.0))))
    tensors = {"router": torch.ones(4, 16) * torch.tensor([[2.0], [2.5], [3.0], [2.25]])}
    for e in range(4):
        for name in ("gate", "up", "down"):
            tensors[f"e{e}.{name}"] = torch.full((16, 16), 0.01 * (e + 1)).to(rt.dtype)
    part.bind({name: t.cuda() for name, t in tensors.items()}, rt)
    out = torch.empty(1, 16, dtype=torch.float32).cuda()
    rt.ops.advance(torch.zeros(1, 16).cuda(), part.forward(torch.ones(1, 16, dtype=rt.dtype).cuda(), SimpleNamespace()), out)
    want = plain.clamped_unit(torch.ones(1, 16, dtype=F), {n: tensors["e2." + n].double() for n in ("gate", "up", "down")}, 9.0)
    close(out, want, dtype, scale=float(want.max()), loose=2e-2)


def paged(c, r, contexts, lengths, page, dtype, seed):
    """Pages that hold rows [c | r] (one list of rows a request), in random order, and the step's device arrays."""
    total = [a + b for a, b in zip(contexts, lengths)]
    counts = [-(-t // page) for t in total]
    order = torch.randperm(sum(counts) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    k = torch.full((len(order), page, c[0].shape[1]), 9.0, dtype=dtype)      # what no key of these requests is stands out
    v = torch.full((len(order), page, r[0].shape[1]), 9.0, dtype=dtype)
    table = torch.full((len(lengths), max(counts)), -1, dtype=torch.int32)
    cursor = 0
    for request, count in enumerate(counts):
        for index in range(count):
            place = order[cursor]
            cursor += 1
            table[request, index] = place
            rows = slice(index * page, min((index + 1) * page, total[request]))
            k[place, :rows.stop - rows.start] = c[request][rows]
            v[place, :rows.stop - rows.start] = r[request][rows]
    kv = SimpleNamespace(group=0, num_pages=len(order), page_size=page, k=k.cuda(), v=v.cuda())
    ctx = step_of(lengths)
    ctx.positions = torch.cat([torch.arange(a, a + b) for a, b in zip(contexts, lengths)]).int().cuda()
    ctx.block_tables = [table.cuda()]
    ctx.context_lens = torch.tensor(contexts, dtype=torch.int32).cuda()
    ctx.query_lens = torch.tensor(lengths, dtype=torch.int32).cuda()
    ctx.host = SimpleNamespace(query_lens=np.asarray(lengths), context_lens=np.asarray(contexts), num_single=ctx.num_single)
    return ctx, kv


@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(2, 64, 32, 64, 64), (3, 128, 64, 128, 96), (1, 8, 8, 8, 8),
                                                     (2, 40, 16, 72, 24), (2, 72, 64, 40, 136), (1, 128, 16, 96, 32)])
@pytest.mark.parametrize("window", [0, 1, 130, 256])
def test_expanded_prompt_attention_and_one_key_that_stands_out(heads, dim, rot, vdim, rank, window):
    """Portions over contexts of their own (none, a few keys, several tiles), with single tokens before them in the step;
    in every request one key is turned along one query so that it takes nearly all the weight: the window's first key,
    the one before it (which must not show), one far back, one at a page's and at a tile's edge, the query's own."""
    rt = runtime("bfloat16")
    assert rt.ops.expands_latents(dim, rot, vdim, rank)
    page, scale = 16, 0.3 / (dim + rot) ** 0.5 * 8
    lengths, contexts = [1, 150, 40, 260], [5, 0, 300, 7]
    total = [a + b for a, b in zip(lengths, contexts)]
    w_uk, w_uv = (rand(heads, dim, rank, scale=rank ** -0.5, seed=1).bfloat16(),
                  rand(heads, vdim, rank, scale=rank ** -0.5, seed=2).bfloat16())
    sink, gates = torch.tensor([4.0, -2.0, 0.5])[:heads], rand(sum(lengths), heads * vdim, scale=2.0, seed=3)
    base = 300.0
    freq = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F)
    rotation = SimpleNamespace(inv_freq=freq.float().cuda(), magnitude=1.0, interleaved=True, dims=rot)
    for edge in range(5):
        q = rand(sum(lengths), heads, dim + rot, seed=4)
        c = [rand(t, rank, seed=20 + i).bfloat16() for i, t in enumerate(total)]
        r = [rand(t, rot, seed=30 + i).bfloat16() for i, t in enumerate(total)]
        at = np.concatenate([[0], np.cumsum(lengths)])
        turned = [plain.rotate_pairs(q[at[i]:at[i + 1], :, dim:].double(), torch.arange(contexts[i], total[i]), base)
                  for i in range(len(lengths))]
        for i in range(1, len(lengths)):
            t = lengths[i] - 1
            last = total[i] - 1
            place = [last, 2, min(128, last), min(last, 47), 0][edge]
            if window and edge >= 3:
                place = max(0, last - window + (1 if edge == 3 else 0))       # just inside, just outside
            r[i][place] = (turned[i][t, 0] * 40.0 / turned[i][t, 0].norm()).bfloat16()
        # the row at each such place, as the query sees it
        want = []
        for i in range(len(lengths)):
            plain_keys = torch.einsum("hdr,tr->thd", w_uk.double(), c[i].double())
            values = torch.einsum("hdr,tr->thd", w_uv.double(), c[i].double())
            pos = torch.arange(contexts[i], total[i]).view(-1, 1)
            key = torch.arange(total[i]).view(1, -1)
            seen = key <= pos
            if window:
                seen &= key > pos - window
            mine = []
            for h in range(heads):
                scores = (q[at[i]:at[i + 1], h, :dim].double() @ plain_keys[:, h].T + turned[i][:, h] @ r[i].double().T) * scale
                scores = scores.masked_fill(~seen, -np.inf)
                top = torch.maximum(scores.max(-1, keepdim=True).values, sink[h].double())
                weights = torch.exp(scores - top)
                mine.append(weights @ values[:, h] / (weights.sum(-1, keepdim=True) + torch.exp(sink[h].double() - top)))
            want.append(torch.stack(mine, 1))
        want = torch.cat(want) * torch.sigmoid(gates.double()).view(-1, heads, vdim)
        ctx, kv = paged(c, r, contexts, lengths, page, torch.bfloat16, seed=edge)
        plan = {name: torch.from_numpy(array).cuda() for name, array in rt.ops.plan_latent_prompt(ctx.host, window).items()}
        out = torch.full((sum(lengths), heads * vdim), 5.0, dtype=torch.bfloat16).cuda()
        w_kv = torch.cat([w_uk, w_uv], 1).reshape(-1, rank).cuda()
        rt.ops.latent_prompt(q.reshape(sum(lengths), -1).cuda(), out, ctx, kv, rotation, plan, w_kv, sink.cuda(), heads, dim,
                             rot, vdim, rank, scale, window=window, gate=gates.cuda())
        rt.ops.check_errors()
        assert (out[:1] == 5.0).all()                     # the single token's row is somebody else's
        close(out[1:].view(-1, heads, vdim), want[1:], "bfloat16", scale=1.0, loose=6e-2)


def test_heads_that_are_expanded_in_turns(monkeypatch):
    """A small bound on the expanded rows: the heads come two at a time and the last alone."""
    from cloud_inference_from_scratch_b200.native import ops as ops_module

    heads, dim, rot, vdim, rank, page = 5, 32, 16, 24, 40, 16
    lengths, contexts = [200], [100]
    q, c, r = rand(200, heads * (dim + rot), seed=1), [rand(300, rank, seed=2).bfloat16()], [rand(300, rot, seed=3).bfloat16()]
    w_kv = rand(heads * (dim + vdim), rank, scale=0.2, seed=4).bfloat16().cuda()
    rotation = SimpleNamespace(inv_freq=torch.ones(rot // 2).cuda(), magnitude=1.0, interleaved=True, dims=rot)
    results = []
    for limit in (1 << 28, 2 * 384 * 2 * (dim + vdim) + 10):
        monkeypatch.setattr(ops_module, "LATENT_PROMPT_BYTES", limit)
        rt = runtime("bfloat16")
        ctx, kv = paged(c, r, contexts, lengths, page, torch.bfloat16, seed=0)
        plan = {name: torch.from_numpy(array).cuda() for name, array in rt.ops.plan_latent_prompt(ctx.host).items()}
        out = torch.empty(200, heads * vdim, dtype=torch.bfloat16).cuda()
        before = rt.ops.launches
        rt.ops.latent_prompt(q.cuda(), out, ctx, kv, rotation, plan, w_kv, None, heads, dim, rot, vdim, rank, 0.2)
        results.append((out.cpu(), rt.ops.launches - before))
        rt.ops.check_errors()
    assert results[1][1] - results[0][1] == 2              # three turns instead of one
    close(results[1][0], results[0][0], "bfloat16", scale=1.0, loose=1e-2)


@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_a_far_key_that_stands_out_in_the_whole_model(folders, name, tmp_path):
    """Queries and keys scaled until scores differ by tens: what a token reads is one key, wherever it lies; in prompts
    and in decoding, with keys at page borders and in the first positions among them."""
    import safetensors.torch

    folder = folders[name, "float32"]
    sharp = tmp_path / "sharp"
    sharp.mkdir()
    (sharp / "config.json").write_text((Path(folder) / "config.json").read_text())
    tensors = safetensors.torch.load_file(str(Path(folder) / "model.safetensors"))
    for key in list(tensors):
        if key.endswith("mix.uq") or key.endswith("dkv.norm"):
            tensors[key] = tensors[key] * 3.0
    safetensors.torch.save_file(tensors, str(sharp / "model.safetensors"))
    requests = requests_for(CONFIGS[name], [140, 90], seed=700)
    for steps in (trace_whole(requests), trace_tail(requests, tail=60), trace_mixed(requests, seed=2, live_limit=2)):
        core = core_for(sharp, "float32", PAGE[name], 320 // PAGE[name], slots=2)
        check(sharp, run_trace(core, steps), "float32", gate=2e-3)


# ------------------------------------------------------------------ the public entry point and the replay program
@pytest.mark.parametrize("name", ["mixed", "tiles"])
def test_greedy_generation_through_the_engine(folders, name):
    from cloud_inference_from_scratch_b200 import generate

    folder = folders[name, "float32"]
    raw, tensors = plain.read_folder(folder)
    prompts = [random_tokens(raw["vocab"], n, 300 + n) for n in (5, 19, 33)]
    want = [plain.greedy(raw, tensors, prompt, 8) for prompt in prompts]
    results = generate(folder, prompts, max_output_tokens=8, dtype="float32", block_size=4, kv_cache_blocks=64,
                       prefill_chunk_size=16, max_batched_tokens=40)
    assert [result.token_ids for result in results] == want


def test_bfloat16_generation_with_graphs_and_a_long_prompt_among_short_ones(folders):
    """Decode steps run from captured graphs (padded batches of three in four rows, whose state must not move), a long
    prompt arrives in portions that run on expanded keys; every token lies within rounding of the plain model's best."""
    from cloud_inference_from_scratch_b200 import generate

    folder = folders["tiles", "bfloat16"]
    raw, tensors = plain.read_folder(folder)
    prompts = [random_tokens(raw["vocab"], n, 400 + n) for n in (7, 230, 64)]
    results = generate(folder, prompts, max_output_tokens=12, dtype="bfloat16", block_size=16, kv_cache_blocks=64,
                       prefill_chunk_size=96, max_batched_tokens=128)
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == 12
        logits = plain.forward(raw, tensors, prompt + result.token_ids).numpy()
        for index, token in enumerate(result.token_ids):
            row = logits[len(prompt) + index - 1]
            assert row[token] >= row.max() - 0.15 * logits.std(), f"token {index} of {result.token_ids}"


def test_the_replay_program_on_a_bozevik_folder(folders, tmp_path):
    folder = folders["narrow", "float32"]
    requests = requests_for(CONFIGS["narrow"], [9, 30], seed=500)
    steps = trace_mixed(requests, seed=4, live_limit=2)
    out = tmp_path / "out"
    done = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                           "--max-tokens", "128"], input="\n".join(json.dumps(step) for step in steps) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done")] == [f"done {s['step']}" for s in steps]
    position = {rid: 0 for rid in requests}
    for step in steps:
        rows = np.fromfile(out / f"{step['step']}.f32", dtype="<f4").reshape(-1, CONFIGS["narrow"]["vocab"])
        row = 0
        for entry in step["entries"]:
            ref = plain_logits(folder, requests[entry["id"]])
            for place in entry["want"]:
                assert np.abs(rows[row] - ref[position[entry["id"]] + place]).max() <= 2e-4 * ref.std()
                row += 1
            position[entry["id"]] += len(entry["tokens"])
        assert row == len(rows)
