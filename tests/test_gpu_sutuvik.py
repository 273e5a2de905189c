"""The Sutuvik design in the engine against the plain implementation of ``plain_sutuvik.py``: each mechanism alone,
whole prompts against decoding, portions down to two tokens, unequal batches, pages and state slots that are used
again, far keys and keys at page edges, first tokens, long decoding, sizes of every kind, and greedy generation through
the public entry point."""

import json
import math
import subprocess
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_sutuvik as plain
from helpers import peak_tokens, random_tokens, replay, requests_in, trace_mixed, trace_portions, trace_tail, trace_whole

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
F = torch.float64

# worst |logit difference| of a row over the standard deviation of the request's reference logits
GATE = {"float32": 2e-4, "bfloat16": 0.12}


# ------------------------------------------------------------------ configurations
def biased(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.4, coef=0.25, every=11, v_mix=True):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
                                             q_temp=dict(coef=coef, every=every), v_mix=v_mix))


def rotated(heads=4, kv_heads=2, dim=16, vdim=24, dims=8, scale=0.5, softcap=8.0, base=1000.0, scaling=True, v_mix=True):
    rot = dict(base=base, dims=dims)
    if scaling:
        rot["scaling"] = dict(factor=4.0, low=1.0, high=3.0, original=64)
    return dict(type="attention_2", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
                                               softcap=softcap, rot=rot, v_mix=v_mix))


def mamba(heads=4, vdim=12, state=20, groups=2, conv=4, norm_groups=2):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups))


def moe(layer, ff=16, experts=6, top=2, groups=3, keep=2):
    return dict(layer, mlp=dict(kind="moe", expert=dict(ff=ff),
                                router=dict(experts=experts, top=top, groups=dict(count=groups, keep=keep))))


def bare(layer):
    return dict(layer, mlp=None)


def config(layers, width=64, vocab=211, taps=3, side=8, groups=2, eps=1e-5, scale=0.6):
    return dict(architecture="Sutuvik", vocab=vocab, width=width, logit_scale=scale, norm=dict(eps=eps, groups=groups),
                canon=dict(taps=taps), token_side=dict(dim=side), layers=list(layers))


CONFIGS = {
    # all three mixers, values mixed over both kinds of attention, value sizes unlike key sizes, layers without
    # feed-forward
    "mixed": config([moe(rotated()), bare(mamba()), moe(biased()), bare(rotated(heads=2, dim=24, dims=24, scaling=False)),
                     moe(mamba(heads=6, groups=3, conv=2, norm_groups=3))]),
    # one of everything: one head, one group, one expert, one tap in front of the mixers, one norm group, one tap in the
    # recurrence's convolution
    "single": config([moe(mamba(heads=1, vdim=16, state=16, groups=1, conv=1, norm_groups=1), ff=24, experts=1, top=1, groups=1, keep=1),
                      moe(biased(heads=1, kv_heads=1, dim=16, vdim=16, every=1, v_mix=False), experts=4, top=4, groups=1, keep=1),
                      bare(rotated(heads=1, kv_heads=1, dim=8, vdim=8, dims=2, v_mix=False))],
                     width=48, vocab=130, taps=1, groups=1, side=16, scale=1.0),
    # sizes that are no multiples of eight; values larger than keys; many norm groups; a long filter; the first layer
    # with mixed values is not the first with attention
    "narrow": config([moe(biased(heads=6, kv_heads=2, dim=10, vdim=7, v_mix=False), ff=10, experts=9, top=4, groups=3, keep=2),
                      bare(biased(heads=3, kv_heads=1, dim=6, vdim=14)),
                      moe(mamba(heads=9, vdim=5, state=11, groups=3, conv=5, norm_groups=5), ff=7, experts=4, top=1, groups=4, keep=1),
                      moe(rotated(heads=2, kv_heads=1, dim=14, vdim=14, dims=6, softcap=3.0))],
                     width=36, vocab=77, taps=6, side=5, groups=12, eps=1e-6, scale=1.3),
    # sizes that the tensor-core kernels take: heads of 64 and 32 with values larger and smaller; a state of
    # more than one tile
    "tiles": config([moe(rotated(heads=8, kv_heads=2, dim=64, vdim=96, dims=32, scale=0.08, softcap=20.0), ff=32, experts=8, top=3, groups=4, keep=2),
                     bare(mamba(heads=4, vdim=64, state=80, groups=1, conv=4, norm_groups=4)),
                     moe(biased(heads=4, kv_heads=2, dim=32, vdim=96, scale=0.2, every=40), ff=32, experts=8, top=2, groups=2, keep=1),
                     bare(biased(heads=2, kv_heads=2, dim=64, vdim=32, scale=0.15, v_mix=False))],
                    width=128, side=24, taps=4, groups=4),
    # no attention at all: no pages, only state slots
    "recurrent": config([moe(mamba(heads=2, vdim=16, state=16, groups=1)), bare(mamba(heads=8, vdim=8, state=24, groups=8))],
                        width=32, vocab=90),
}
PAGE = {"mixed": 4, "single": 16, "narrow": 8, "tiles": 16, "recurrent": 8}
# N(0, 0.05) weights leave sinks, filters, rates and biases close to nothing
SCALES = {"canon1": 6.0, "mix.conv": 8.0, "dt_bias": 30.0, "A_log": 25.0, "sink": 40.0, "vmix": 8.0, "side.embed": 20.0,
          "side.gate": 4.0, "mix.q": 2.0, "mix.k": 2.0, "mix.v": 2.0, "mix.g": 5.0, "mix.in": 3.0, "mlp.router": 8.0,
          "correction": 12.0, "mlp.e": 3.0}
# the bfloat16 runs of whole models let the stored correction alone choose the experts (the router still sets the
# weights): else some token has two experts within bfloat16 rounding of each other and goes either way; and they
# shrink the side input, which divides something small by its own size
SCALES_BF16 = dict(SCALES, correction=400.0, **{"mlp.router": 4.0, "side.norm": 0.3, "mix.q": 1.4, "mix.k": 1.4})


def make_model(folder, raw, seed, std=0.05, scales=None):
    from cloud_inference_from_scratch_b200.weights import write_random_model

    return write_random_model(folder, raw, seed, std=std, scales=scales or SCALES)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("sutuvik")
    out = {}
    for index, (name, raw) in enumerate(CONFIGS.items()):
        out[name, "float32"] = make_model(root / name, raw, 5 + index)
        out[name, "bfloat16"] = make_model(root / (name + "-fixed"), raw, 5 + index, scales=SCALES_BF16)
    return out


def core_for(folder, dtype, page, pages, slots=4, step_tokens=0):
    from cloud_inference_from_scratch_b200.engine.core import build_core

    return build_core(folder, dtype=dtype, page_size=page, num_pages=pages, max_requests=slots,
                      max_model_len=pages * page, max_tokens_per_step=step_tokens)


PLAIN_LOGITS = {}


def plain_logits(folder, tokens, noise=None):
    key = (str(folder), tuple(tokens), noise)
    if key not in PLAIN_LOGITS:
        raw, tensors = plain.read_folder(folder)
        PLAIN_LOGITS[key] = plain.forward(raw, tensors, tokens, noise=noise).numpy()
    return PLAIN_LOGITS[key]


def check(folder, got, dtype, gate=None):
    """Every row against the plain model run on the whole request.  In bfloat16 (float32 has held every row to a far
    sharper gate) a position may also be off by four times what the plain logits move there in one of eight runs
    with the inputs of products and the cached rows moved by up to the rounding of bfloat16: a norm of something
    small blows rounding up at a few positions, and at a few only."""
    limit = gate or GATE[dtype]
    worst = 0.0
    for rid, tokens in got["fed"].items():
        ref = plain_logits(folder, tokens)
        rows = got["logits"][rid]
        assert sorted(rows) == list(range(len(tokens))), f"{rid}: positions missing"
        mine = np.stack([rows[p] for p in range(len(tokens))])
        errors = np.abs(mine - ref).max(axis=1) / ref.std()
        allowed = np.full(len(tokens), limit)
        if dtype == "bfloat16":
            drawn = np.stack([plain_logits(folder, tokens, noise) for noise in range(8)])
            allowed = np.maximum(limit, 4.0 * np.abs(drawn - ref).max(axis=(0, 2)) / ref.std())
            assert (allowed > 2 * limit).sum() <= max(4, len(tokens) // 6), f"{rid}: rounding decides too many rows"
        worst = max(worst, float(errors.max()))
        wrong = errors > allowed
        assert not wrong.any(), (
            f"{rid}: first wrong position {int(np.argmax(wrong))} of {len(tokens)}, error {errors[np.argmax(wrong)]:.3e}")
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
    # lengths: one token, two, a page's edge and one past it, several pages, one and two of the recurrence's chunks
    requests = requests_for(CONFIGS[name], [1, 2, page, page + 1, 23, 64, 65, 141], seed=10)
    for steps in (trace_whole(requests), trace_tail(requests, tail=40), trace_portions(requests),
                  trace_mixed(requests, seed=3, live_limit=3)):
        # a pool that holds what is live and no more, and three slots: pages and slots come back
        pages = -(-peak_tokens(steps, round_to=page) // page) + 1
        core = core_for(folder, dtype, page, pages, slots=3)
        check(folder, run_trace(core, steps), dtype)
        assert core.cache.free_pages(0) == core.cache.total_pages(0)


def drawn_configuration(seed):
    """A configuration drawn from the whole space of sizes: widths, any layer kind in any order, head counts, key and
    value sizes (multiples of 8 and 16 and others, above and below what the tensor-core kernels take), rotated parts
    from two elements to the whole head with and without scaled frequencies, caps, temperatures, filters, states and
    groups of every size, experts from one to many in one group or several, layers without feed-forward."""
    import random

    rng = random.Random(seed)
    layers, kv_width = [], rng.choice([(2, 16), (1, 40), (4, 8), (2, 64), (1, 128), (2, 80)])
    for _ in range(rng.randint(2, 5)):
        kind = rng.choice(["biased", "rotated", "mamba"])
        if kind == "mamba":
            groups, per = rng.choice([1, 2, 3]), rng.choice([1, 2, 4])
            vdim = rng.choice([4, 16, 32, 64, 72, 128])
            layer = mamba(groups * per, vdim, rng.choice([3, 16, 48, 64, 100, 128, 200]), groups, rng.choice([1, 2, 3, 4, 7]),
                          rng.choice([1, groups, groups * per]))
        else:
            mixes = rng.random() < 0.7
            kv, vdim = kv_width if mixes else (rng.choice([1, 2, 3]), rng.choice([8, 16, 36, 64, 144]))
            dim, group = rng.choice([8, 16, 24, 32, 64, 80, 128]), rng.choice([1, 2, 3, 9])
            scale = rng.choice([0.4, 1.0, 2.5]) / dim ** 0.5
            if kind == "biased":
                layer = biased(kv * group, kv, dim, vdim, scale, rng.choice([0.1, 0.7]), rng.choice([1, 7, 64, 1000]), mixes)
            else:
                layer = rotated(kv * group, kv, dim, vdim, rng.choice([2, dim // 2, dim]) // 2 * 2,
                                scale * rng.choice([1.0, 4.0]), rng.choice([1.5, 12.0, 60.0]),
                                rng.choice([100.0, 10000.0]), rng.random() < 0.7, mixes)
        if rng.random() < 0.7:
            groups, per = rng.choice([1, 2, 4]), rng.choice([1, 2, 5])
            keep = rng.randint(1, groups)
            layer = moe(layer, rng.choice([8, 16, 24, 40]), groups * per, rng.randint(1, keep * per), groups, keep)
        else:
            layer = bare(layer)
        layers.append(layer)
    norm_groups = rng.choice([1, 2, 3, 8, 24])
    width = norm_groups * rng.choice([n for n in range(2, 260) if 48 <= n * norm_groups <= 264 and n * norm_groups % 4 == 0])
    return config(layers, width=width, vocab=rng.choice([50, 211, 450]), taps=rng.choice([1, 2, 3, 4, 5]),
                  side=rng.choice([3, 8, 16, 40]), groups=norm_groups, eps=rng.choice([1e-6, 1e-5]),
                  scale=rng.choice([0.25, 1.0, 2.0]))


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_drawn_configurations(seed, tmp_path):
    raw = drawn_configuration(seed)
    requests = requests_for(raw, [1, 2, 37, 150], seed=seed)
    for dtype, scales, gate in (("float32", SCALES, 4e-4), ("bfloat16", SCALES_BF16, 0.2)):
        folder = make_model(tmp_path / dtype, raw, 100 + seed, scales=scales)
        for steps in (trace_whole(requests), trace_mixed(requests, seed=seed, live_limit=3)):
            pages = -(-peak_tokens(steps, round_to=16) // 16) + 1
            core = core_for(folder, dtype, 16, pages, slots=3)
            check(folder, run_trace(core, steps), dtype, gate=gate)


def test_float32_rows_do_not_depend_on_the_cut_or_the_batch(folders):
    """The same position through four cuttings: equal to rounding of the order of additions at most."""
    requests = requests_for(CONFIGS["mixed"], [50, 31, 77], seed=40)
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


def test_long_decoding(folders):
    """160 tokens decoded one by one after a short prompt: state, histories and temperature are carried for every
    token, over many pages."""
    for name in ("mixed", "narrow"):
        requests = requests_for(CONFIGS[name], [170, 165], seed=70)
        steps = trace_tail(requests, tail=160)
        for dtype in ("float32", "bfloat16"):
            core = core_for(folders[name, dtype], dtype, PAGE[name], 400 // PAGE[name], slots=2)
            check(folders[name, dtype], run_trace(core, steps), dtype)


def test_a_state_slot_that_is_used_again_starts_from_zero(folders):
    """One slot only: every request inherits the slot of the one before it."""
    for name in ("mixed", "recurrent"):
        requests = requests_for(CONFIGS[name], [30, 8, 19], seed=90)
        core = core_for(folders[name, "float32"], "float32", PAGE[name], 16, slots=1)
        check(folders[name, "float32"], run_trace(core, trace_portions(requests)), "float32")


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


def step_of(lengths, contexts, page, dtype, heads=1, dim=8, vdim=8, seed=0, slots=None, active=None):
    """A step of requests that hold ``contexts`` tokens and bring ``lengths``, over empty pools."""
    total = [c + n for c, n in zip(contexts, lengths)]
    pages_per = [-(-t // page) for t in total]
    order = torch.randperm(sum(pages_per) + 2, generator=torch.Generator().manual_seed(seed)).tolist()
    table = torch.full((len(lengths), max(pages_per)), -1, dtype=torch.int32)
    cursor = 0
    for r, count in enumerate(pages_per):
        table[r, :count] = torch.tensor(order[cursor:cursor + count], dtype=torch.int32)
        cursor += count
    kv = SimpleNamespace(group=0, num_pages=len(order), page_size=page,
                         k=torch.zeros(len(order), heads, page, dim, dtype=dtype).cuda(),
                         v=torch.zeros(len(order), heads, page, vdim, dtype=dtype).cuda())
    singles = 0
    while singles < len(lengths) and lengths[singles] == 1:
        singles += 1
    starts = np.concatenate([[0], np.cumsum(lengths)]).astype(np.int32)
    ints = lambda values: torch.tensor(values, dtype=torch.int32).cuda()  # noqa: E731
    ctx = SimpleNamespace(
        positions=torch.cat([torch.arange(c, c + n) for c, n in zip(contexts, lengths)]).int().cuda(),
        request_of_token=torch.cat([torch.full((n,), r) for r, n in enumerate(lengths)]).int().cuda(),
        block_tables=[table.cuda()], num_requests=len(lengths), num_single=singles, extras={},
        context_lens=ints(contexts), query_lens=ints(lengths), query_start=torch.from_numpy(starts).cuda(),
        slots=ints(slots if slots is not None else list(range(len(lengths)))),
        request_active=ints(active if active is not None else [1] * len(lengths)),
        host=SimpleNamespace(query_lens=np.asarray(lengths, dtype=np.int32), num_single=singles,
                             num_requests=len(lengths), query_start=starts))
    return ctx, kv


def plan_into(ctx, rt, group):
    plan = rt.ops.plan_attention(ctx.host, group)
    if plan:
        ctx.extras[("attention", group)] = {name: torch.from_numpy(np.asarray(a)).cuda() for name, a in plan.items()}


def updates_for(rows, width, rt):
    """Every kind of pending update with the plain value that joins the stream."""
    from cloud_inference_from_scratch_b200.lazy import NormedUpdate, Partials, WeightedTerms

    first, second = rand(rows, width, seed=4), rand(rows, width, seed=5)
    both = torch.stack([first, second]).cuda().contiguous()
    gain, share = 1 + rand(width, scale=0.3, seed=6), rand(rows, 3, seed=7)
    return [(None, torch.zeros(rows, width, dtype=F)), (first.cuda(), first.double()),
            (Partials(both, 2, rows, width, None), (first + second).double()),
            (first.to(rt.dtype).cuda(), first.to(rt.dtype).double()),
            (WeightedTerms(torch.cat([first, second, first * second], 1).cuda(), share.cuda()),
             (torch.stack([first, second, first * second], 1).double() * share.double().unsqueeze(-1)).sum(1)),
            (NormedUpdate(first.cuda(), gain.cuda(), 1e-5), plain.rms(first.double(), 1e-5) * gain.double())]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,groups", [(40, 1), (36, 3), (36, 12), (192, 6), (2048, 4), (9000, 5), (640, 40), (21, 7)])
def test_norm_in_groups_with_every_kind_of_update(dtype, width, groups):
    """Groups of very different size (a norm over the whole row, or over the wrong part, shows at once); all rows,
    selected rows, the stream's own rows rounded, and the stream normalised in place."""
    rt = runtime(dtype)
    rows, eps = 5, 1e-5
    stream = rand(rows, width, seed=1) * torch.logspace(-2, 2, groups).repeat_interleave(width // groups)
    gain = 1 + rand(width, scale=0.2, seed=2)
    for update, added in updates_for(rows, width, rt):
        total = stream.double() + added
        want = plain.group_norm(total, gain.double(), eps, groups)
        residual, out = stream.clone().cuda(), torch.empty(rows, width, dtype=rt.dtype).cuda()
        rt.ops.group_norm(residual, update, gain.cuda(), eps, groups, out)
        close(residual, total, "float32", scale=1.0, tight=2e-5)
        close(out, want, dtype, scale=1.0, tight=1e-4)
        chosen = torch.tensor([4, 0, 4], dtype=torch.int32).cuda()
        residual, picked = stream.clone().cuda(), torch.empty(3, width, dtype=rt.dtype).cuda()
        rt.ops.group_norm(residual, update, gain.cuda(), eps, groups, picked, chosen)
        assert torch.equal(residual.cpu(), stream)
        close(picked, want[[4, 0, 4]], dtype, scale=1.0, tight=1e-4)
        residual, own = stream.clone().cuda(), torch.empty(rows, width, dtype=rt.dtype).cuda()
        rt.ops.group_norm(residual, update, None, 0.0, 1, own)
        close(own / total.abs().max().float().cuda(), total / total.abs().max(), dtype, scale=1.0, tight=2e-6)
        residual = stream.clone().cuda()
        rt.ops.group_norm(residual, None, gain.cuda(), eps, groups, residual)
        close(residual, plain.group_norm(stream.double(), gain.double(), eps, groups), "float32", scale=1.0, tight=1e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,groups,taps", [(36, 3, 3), (64, 2, 1), (96, 4, 2), (33, 1, 4), (128, 1, 16), (2048, 8, 5)])
def test_norm_and_input_convolution_over_requests_that_come_in_pieces(dtype, width, groups, taps):
    """Requests of several lengths, cut into portions (longer and shorter than the filter) and single tokens, against
    the whole sequences at once; a request that is not active leaves its history alone."""
    rt = runtime(dtype)
    eps = 1e-5
    gain, w = 1 + rand(width, scale=0.2, seed=2), rand(width, taps, scale=0.7, seed=3)
    lengths = [23, 9, 40]
    streams = [rand(n, width, seed=10 + r) for r, n in enumerate(lengths)]
    want = []
    for x in streams:
        h = plain.group_norm(x.double(), gain.double(), eps, groups)
        want.append(h + plain.causal_conv(h, w.double()))
    pad = 4                                            # the history lies behind other numbers of the slot
    floats = (taps - 1) * width
    state = torch.zeros(4, pad + floats).cuda() if taps > 1 else None
    history = state[:, pad:] if taps > 1 else None
    done = [0, 0, 0]
    for portions in ([1, 1, 1], [5, 1, 2], [2, 3, 1], [1, 1, 1], [13, 2, 30], [1, 1, 1]):
        order = sorted(range(3), key=lambda r: portions[r] != 1)       # single tokens lead a step
        sizes = [min(portions[r], lengths[r] - done[r]) for r in order]
        residual = torch.cat([streams[r][done[r]:done[r] + n] for r, n in zip(order, sizes)]).cuda()
        update = rand(*residual.shape, seed=77).cuda()
        for active in ([0, 0, 0], [1, 1, 1]):           # first as padding: the histories must stay
            ctx, _ = step_of(sizes, [done[r] for r in order], 16, rt.dtype, slots=[(2, 0, 3)[r] for r in order], active=active)
            out = torch.empty(residual.shape, dtype=rt.dtype).cuda()
            moving = (residual - update).contiguous()
            before = state.clone() if taps > 1 else None
            rt.ops.group_norm_conv(moving, update, gain.cuda(), eps, groups, w.cuda(), history, out, ctx)
            rt.ops.check_errors()
            close(moving, residual, "float32", scale=1.0, tight=1e-6)
            if taps > 1 and not active[0]:
                assert torch.equal(state, before)
            row = 0
            for r, n in zip(order, sizes):
                close(out[row:row + n], want[r][done[r]:done[r] + n], dtype, scale=1.0, loose=5e-2, tight=1e-4)
                row += n
        for r, n in zip(order, sizes):
            done[r] += n
    if taps > 1:
        assert state[:, :pad].abs().max() == 0 and state[1].abs().max() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gated_norm_in_groups_and_the_side_gate(dtype):
    rt = runtime(dtype)
    rt.ops.require_grouped()
    for width, groups in ((48, 3), (33, 1), (4096, 8), (60, 20)):
        y, wide = rand(6, width, scale=3.0, seed=1), rand(6, width + 7, scale=2.0, seed=2)
        gain = 1 + rand(width, scale=0.3, seed=3)
        out = torch.empty(6, width, dtype=rt.dtype).cuda()
        rt.ops.gated_group_norm(y.cuda(), wide.cuda()[:, 7:], gain.cuda(), 1e-5, groups, out)
        want = plain.group_norm(y.double() * plain.silu(wide[:, 7:].double()), gain.double(), 1e-5, groups)
        close(out, want, dtype, scale=1.0, loose=5e-2, tight=2e-5)
    table, ids = rand(11, 40, seed=4).to(rt.dtype), torch.tensor([3, 10, 0, 3], dtype=torch.int32)
    z = rand(4, 9, scale=3.0, seed=5)
    out = torch.empty(4, 9, dtype=rt.dtype).cuda()
    rt.ops.side_gate(z.cuda(), ids.cuda(), table.cuda(), 18, out)
    rt.ops.check_errors()
    close(out, plain.gelu_tanh(z.double()) * table[ids.long()][:, 18:27].double(), dtype, scale=1.0, loose=3e-2, tight=1e-5)
    # far below zero the result is nearly nothing, but what there is must be right to nearly float32's last digits
    z = torch.linspace(-5.0, -2.0, 36).view(4, 9)
    rt.ops.side_gate(z.cuda(), ids.cuda(), torch.ones(11, 40).to(rt.dtype).cuda(), 18, out)
    exact = plain.gelu_tanh(z.double())
    close(out.double().cpu() / exact, torch.ones(4, 9), dtype, scale=1.0, loose=1e-2, tight=1e-5)


def rotation_of(rot):
    return SimpleNamespace(inv_freq=plain.wavelength_frequencies(rot).float().cuda(), magnitude=1.0, interleaved=True,
                           dims=rot["dims"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim,group", [(16, 24, 2), (64, 32, 4), (32, 64, 1), (20, 12, 3), (128, 128, 2), (48, 80, 9), (8, 144, 2)])
def test_biased_attention_far_keys_edges_and_a_sink(dtype, dim, vdim, group):
    """Per-head norm with gains, a temperature, slopes, a sink and a gate per head.  For the last query of a request of
    300 tokens one key at a time (the first, one far back, both sides of a page's edge, its own) is turned along that
    query so that it outweighs the slope's penalty; whole prompt, a portion over cached keys, a single token."""
    rt = runtime(dtype)
    groups, page, eps, n = 2, 16, 1e-5, 300
    heads = groups * group
    scale, coef, every = 6.0 / dim ** 0.5, 0.3, 64
    rt.ops.require_portion_attention(max(dim, vdim))
    width = heads * dim + groups * (dim + vdim)
    q_gain, k_gain = 1 + rand(dim, scale=0.2, seed=3), 1 + rand(dim, scale=0.2, seed=4)
    sink, slopes, gates = rand(heads, scale=3.0, seed=5), plain.head_slopes(heads), rand(n, heads + 3, scale=2.0, seed=6)
    heat = plain.query_temperature(torch.arange(n), coef, every).view(-1, 1, 1)
    shared = heads - 1                     # the head with the smallest slope looks furthest; it reads the last kv head
    for edge in (0, 37, page * 9 - 1, page * 9, n - 1):
        full = rand(n, width, seed=1)
        last = plain.rms(full[n - 1, shared * dim:(shared + 1) * dim].double(), eps) * q_gain.double()
        at = heads * dim + (groups - 1) * dim
        full[edge, at:at + dim] = (last / k_gain.double()).float() * 5.0
        x = full.double()
        q = plain.rms(x[:, :heads * dim].view(n, heads, dim), eps) * q_gain.double() * heat
        k = plain.rms(x[:, heads * dim:heads * dim + groups * dim].view(n, groups, dim), eps) * k_gain.double()
        v = x[:, heads * dim + groups * dim:].view(n, groups, vdim)
        want = plain.attend(q, k, v, scale, sink.double(), slopes=slopes) * torch.sigmoid(gates[:, 3:].double()).unsqueeze(-1)
        for lengths, contexts in (([n], [0]), ([n - 250], [250]), ([1], [n - 1])):
            ctx, kv = step_of([n], [0], page, rt.dtype, groups, dim, vdim, seed=2)
            held = contexts[0]
            q_all = torch.empty(n, heads * dim, dtype=rt.dtype).cuda()
            rt.ops.norm_kv_write(full.cuda(), ctx, kv, heads, groups, dim, vdim, q_gain.cuda(), k_gain.cuda(), False, eps,
                                 q_all, per_head=True, heat=(coef, every))
            step, _ = step_of(lengths, contexts, page, rt.dtype, groups, dim, vdim, seed=2)
            plan_into(step, rt, group)
            out = torch.empty(n - held, heads * vdim, dtype=rt.dtype).cuda()
            rt.ops.attention_penalised(q_all[held:].contiguous(), out, step, kv, heads, groups, dim, vdim, scale, 0, None,
                                       sinks=sink.cuda(), slopes=slopes.float().cuda(), gates=gates.cuda()[held:, 3:])
            rt.ops.check_errors()
            # in bfloat16 a score of 60 carries a rounding of the query and the key of 0.1
            close(out.view(n - held, heads, vdim), want[held:], dtype, scale=1.0, loose=2e-1, tight=1e-4)
        close(q_all.view(n, heads, dim), q, dtype, scale=1.0, loose=4e-2, tight=5e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim,dims,group,cap", [(16, 24, 8, 2, 9.0), (64, 32, 32, 2, 50.0), (20, 12, 20, 1, 4.0), (32, 64, 2, 4, 15.0), (128, 128, 64, 8, 30.0)])
def test_rotated_attention_unit_size_factor_cap_and_one_in_the_denominator(dtype, dim, vdim, dims, group, cap):
    """Rotation with frequencies scaled by wavelength, THEN a norm without gains; a factor per head before the cap;
    single keys turned along the last query so that the cap bites."""
    rt = runtime(dtype)
    groups, page, eps, n = 2, 16, 1e-5, 300
    heads = groups * group
    scale = 2.0 * cap / dim
    rot = dict(base=2000.0, dims=dims, scaling=dict(factor=6.0, low=1.0, high=4.0, original=128))
    rt.ops.require_portion_attention(max(dim, vdim))
    width = heads * dim + groups * (dim + vdim)
    factor = 1 + rand(heads, scale=0.4, seed=7)
    for edge in (0, 37, page * 9 - 1, page * 9, n - 1):
        full = rand(n, width, seed=1)
        at = torch.arange(n)
        q = plain.rms(plain.rotate_pairs(full[:, :heads * dim].double().view(n, heads, dim), at, rot), eps)
        # the key at `edge`, once rotated, points along head 0 of the last query
        full[edge, heads * dim:heads * dim + dim] = plain.rotate_pairs(q[n - 1:, :1], torch.tensor([-edge]), rot)[0, 0].float() * 3.0
        k = plain.rms(plain.rotate_pairs(full[:, heads * dim:heads * dim + groups * dim].double().view(n, groups, dim), at, rot), eps)
        v = full[:, heads * dim + groups * dim:].double().view(n, groups, vdim)
        want = plain.attend(q, k, v, scale, torch.zeros(heads, dtype=F), temps=factor.double(), cap=cap)
        for lengths, contexts in (([n], [0]), ([n - 250], [250]), ([1], [n - 1])):
            ctx, kv = step_of([n], [0], page, rt.dtype, groups, dim, vdim, seed=2)
            held = contexts[0]
            q_all = torch.empty(n, heads * dim, dtype=rt.dtype).cuda()
            rt.ops.norm_kv_write(full.cuda(), ctx, kv, heads, groups, dim, vdim, None, None, False, eps, q_all,
                                 rotation=rotation_of(rot), unit_heads=True, q_factor=factor.cuda())
            step, _ = step_of(lengths, contexts, page, rt.dtype, groups, dim, vdim, seed=2)
            plan_into(step, rt, group)
            out = torch.empty(n - held, heads * vdim, dtype=rt.dtype).cuda()
            rt.ops.attention_penalised(q_all[held:].contiguous(), out, step, kv, heads, groups, dim, vdim, scale, 0, None,
                                       sinks=torch.zeros(heads).cuda(), softcap=cap)
            rt.ops.check_errors()
            close(out.view(n - held, heads, vdim), want[held:], dtype, scale=1.0, loose=1e-1, tight=1e-4)
        close(q_all.view(n, heads, dim), q * factor.double().view(1, -1, 1), dtype, scale=1.0, loose=4e-2, tight=1e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_values_kept_and_blended_and_rows_that_only_pad(dtype):
    """The first layer's values are kept as they are, a later layer's are blended before they are cached; a request
    that is not active writes nothing to the pages."""
    rt = runtime(dtype)
    heads, groups, dim, vdim, page = 2, 2, 8, 12, 4
    n, width = 9, heads * dim + groups * (dim + vdim)
    first, later = rand(n, width, seed=1), rand(n, width, seed=2)
    kept = torch.full((n, groups * vdim), 99.0).cuda()
    share = torch.tensor([0.3]).cuda()
    cut = heads * dim + groups * dim
    for rows, value_share, want in ((first, None, first[:, cut:]), (later, share, 0.7 * later[:, cut:] + 0.3 * first[:, cut:])):
        ctx, kv = step_of([4, 5], [0, 0], page, rt.dtype, groups, dim, vdim, active=[1, 0])
        q = torch.empty(n, heads * dim, dtype=rt.dtype).cuda()
        rt.ops.norm_kv_write(rows.cuda(), ctx, kv, heads, groups, dim, vdim, None, None, False, 1e-5, q, unit_heads=True,
                             first_values=kept, value_share=value_share)
        rt.ops.check_errors()
        assert torch.equal(kept.cpu(), first[:, cut:])
        table = ctx.block_tables[0].cpu()
        page_of = kv.v[int(table[0, 0])].transpose(0, 1).reshape(4, -1)        # the first request's one page
        close(page_of, want[:4], dtype, scale=1.0, loose=2e-2, tight=1e-6)
        for p in table[1].tolist():
            assert p < 0 or (kv.v[p].abs().max() == 0 and kv.k[p].abs().max() == 0)


@pytest.mark.parametrize("heads,groups,dim,vdim", [(2, 1, 12, 20), (4, 2, 64, 64), (3, 3, 128, 40), (8, 1, 100, 32), (2, 2, 5, 33), (2, 1, 200, 130), (6, 2, 16, 8)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_space_recurrence_token_by_token_and_in_chunks(heads, groups, dim, vdim, dtype):
    """Both forms against the plain recurrence, from states that are not zero, with requests of one token, a chunk,
    one more and several chunks, a head that forgets at once, one that keeps everything, and a request that is not
    active (its state must stay).  The 16-bit runtime's chunks run on the tensor cores with every operand as two terms
    and are held to nearly the same gate."""
    rt = runtime(dtype)
    rt.ops.require_ssd()
    lengths = [1, 64, 65, 200, 2]
    tokens, slots = sum(lengths), len(lengths) + 1
    pad = 3 if vdim % 4 else 4             # columns before x: rows that allow 16-byte loads, and rows that do not
    rows = rand(tokens, pad + heads * vdim + 2 * groups * dim, seed=3)
    rates = rand(tokens, heads + 5, scale=1.5, seed=4)
    a_log, bias, skip = rand(heads, seed=5), rand(heads, scale=2.0, seed=6), rand(heads, seed=7)
    a_log[0], a_log[1] = 6.0, -30.0
    x_off, b_off, c_off = pad, pad + heads * vdim, pad + heads * vdim + groups * dim
    x = rows[:, x_off:b_off].double().view(tokens, heads, vdim)
    b = rows[:, b_off:c_off].double().view(tokens, groups, dim)
    c = rows[:, c_off:].double().view(tokens, groups, dim)
    dt = torch.nn.functional.softplus(rates[:, 5:].double() + bias.double(), threshold=1e9)
    start = rand(slots, heads * dim * vdim + 8, seed=9)           # slots wider than the state
    order = [3, 0, 5, 1, 2]
    want, final, first = [], start.double().clone(), 0
    for r, count in enumerate(lengths):
        held = start[order[r], : heads * dim * vdim].double().view(heads, dim, vdim)
        y, last = plain.state_space(x[first:first + count], b[first:first + count], c[first:first + count],
                                    dt[first:first + count], a_log.double(), skip.double(), held)
        want.append(y)
        if r != 2:
            final[order[r], : heads * dim * vdim] = last.reshape(-1)
        first += count
    want = torch.cat(want)
    for chunked in (False, True):
        ctx, _ = step_of(lengths, [0] * len(lengths), 16, torch.float32, slots=order, active=[1, 1, 0, 1, 1])
        plan = {name: torch.from_numpy(a).cuda() for name, a in rt.ops.plan_ssd(ctx.host).items()} if chunked else None
        state = start.clone().cuda()
        out = torch.empty(tokens, heads * vdim).cuda()
        rt.ops.ssd(rows.cuda(), (x_off, b_off, c_off), rates.cuda()[:, 5:], a_log.cuda(), bias.cuda(), skip.cuda(), out, state,
                   ctx, heads, groups, dim, vdim, plan=plan)
        rt.ops.check_errors()
        tight = 3e-5 if dtype == "float32" or not chunked else 3e-4
        close(out.view(tokens, heads, vdim), want, "float32", tight=tight)
        close(state, final, "float32", tight=tight)


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_short_convolution_with_a_bias(taps):
    """A portion, then single tokens, against the whole sequence; columns of a wider row."""
    rt = runtime("float32")
    rt.ops.require_recurrent()
    channels, n = 37, 12
    x, w, bias = rand(n, channels + 6, seed=1), rand(channels, taps, seed=2), rand(channels, seed=3)
    want = plain.silu(plain.causal_conv(x[:, 6:].double(), w.double()) + bias.double())
    state = torch.zeros(3, (taps - 1) * channels + 5).cuda()
    history = state[:, 5:]
    done = 0
    for size in (1, 2, 5, 1, 1, 2):
        ctx, _ = step_of([size], [done], 16, torch.float32, slots=[1])
        out = torch.empty(size, channels).cuda()
        rt.ops.short_conv(x[done:done + size].cuda()[:, 6:], w.cuda(), history, out, ctx, bias=bias.cuda())
        rt.ops.check_errors()
        close(out, want[done:done + size], "float32", scale=1.0, tight=1e-5)
        done += size
    assert state[0].abs().max() == 0 and state[2].abs().max() == 0 and state[:, :5].abs().max() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,top,groups,keep,hidden,ff", [(6, 2, 3, 2, 48, 16), (1, 1, 1, 1, 40, 24), (8, 4, 2, 1, 64, 32), (12, 3, 12, 5, 36, 10), (16, 8, 4, 2, 64, 16)])
def test_routed_experts_sigmoid_scores_and_groups(dtype, experts, top, groups, keep, hidden, ff):
    """Choice scores that are all negative (a group that is left out must count as minus infinity, not as zero), the
    correction steering the choice and not the weights, weights of sum one."""
    from cloud_inference_from_scratch_b200.config import PartSpec
    from cloud_inference_from_scratch_b200.parts import build_part

    rt = runtime(dtype)
    part = build_part("feed_forward", PartSpec("routed_experts", dict(
        hidden_size=hidden, intermediate_size=ff, num_experts=experts, top=top, correction=True, renormalize=True,
        score="sigmoid", groups=(groups, keep), norm_floor=1e-20)))
    tensors = {"router": rand(experts, hidden, scale=0.5, seed=1), "correction": rand(experts, seed=2) - 4.0}
    for e in range(experts):
        tensors[f"e{e}.gate"] = rand(ff, hidden, scale=0.3, seed=10 + e).to(rt.dtype)
        tensors[f"e{e}.up"] = rand(ff, hidden, scale=0.3, seed=40 + e).to(rt.dtype)
        tensors[f"e{e}.down"] = rand(hidden, ff, scale=0.3, seed=70 + e).to(rt.dtype)
    part.bind({name: t.cuda() for name, t in tensors.items()}, rt)
    x = rand(21, hidden, seed=5).to(rt.dtype)
    got = part.forward(x.cuda(), SimpleNamespace())
    rt.ops.check_errors()
    mlp = dict(router=dict(experts=experts, top=top, groups=dict(count=groups, keep=keep)))
    want = plain.routed_feed_forward(x.double(), {name: t.double() for name, t in tensors.items()}, mlp)
    close(got, want, dtype, loose=4e-2, tight=2e-5)
    if keep < groups < experts:      # with every group kept other experts are chosen for some token
        mlp["router"]["groups"]["keep"] = groups
        other = plain.routed_feed_forward(x.double(), {n: t.double() for n, t in tensors.items()}, mlp)
        assert (other - want).abs().max() > 1e-3


# ------------------------------------------------------------------ the public entry point and the replay program
def test_greedy_generation_through_the_engine(folders):
    """Three prompts (a batch of three is padded to four in the captured decode step) through the scheduler."""
    from cloud_inference_from_scratch_b200 import generate

    folder = folders["mixed", "float32"]
    raw, tensors = plain.read_folder(folder)
    prompts = [random_tokens(raw["vocab"], n, 300 + n) for n in (5, 19, 90)]
    want = [plain.greedy(raw, tensors, prompt, 10) for prompt in prompts]
    results = generate(folder, prompts, max_output_tokens=10, dtype="float32", block_size=4, kv_cache_blocks=64,
                       prefill_chunk_size=16, max_batched_tokens=40)
    assert [result.token_ids for result in results] == want


def test_the_replay_program_on_a_sutuvik_folder(folders, tmp_path):
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
    assert math.isfinite(float(ref.std()))
