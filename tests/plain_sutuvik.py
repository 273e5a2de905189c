"""Sutuvik in plain double-precision PyTorch: one function per mechanism, whole sequences only, no cache.

The oracle of the Sutuvik tests.  It shares nothing with the product path: it takes the configuration as the
dictionary that config.json holds and the weights as a dictionary of tensors by their stored names, and walks
a whole sequence at once (the recurrence token by token), so every cutting of a prompt, every batch and every
page layout of the engine is held to the same numbers.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


NOISE = [None]      # a generator: what a 16-bit engine rounds (inputs of products, cached rows) is moved about as much


def rounded(x):
    if NOISE[0] is None:
        return x
    if NOISE[0].initial_seed() == 0:
        return x.to(torch.bfloat16).to(F64)
    return x * (1.0 + (torch.rand(x.shape, generator=NOISE[0], dtype=F64) - 0.5) * 2.0 ** -8)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, gain, eps, groups):
    """Each of ``groups`` equal consecutive parts by its own root mean square; the whole times ``gain``."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape) * gain


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x, w):
    """x [T, C], w [C, taps]: y_t = sum_j w[:, j] x_(t - taps + 1 + j), zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(w[:, j] * padded[j: j + x.shape[0]] for j in range(taps))


def wavelength_frequencies(rot):
    """f_i for i < dims / 2; frequencies of long waves are divided by a factor, those between two wavelengths are
    blended."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return torch.tensor(plain, dtype=F64)
    factor, low, high, original = (float(scaling[key]) for key in ("factor", "low", "high", "original"))
    out = []
    for f in plain:
        length = 2.0 * math.pi / f
        if length < original / high:
            out.append(f)
        elif length > original / low:
            out.append(f / factor)
        else:
            s = (original / length - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return torch.tensor(out, dtype=F64)


def rotate_pairs(x, positions, rot):
    """x [T, heads, size]: elements 2i and 2i + 1 of the first rot.dims of every head turn by position * f_i."""
    dims = int(rot["dims"])
    angle = positions.to(F64).view(-1, 1, 1) * wavelength_frequencies(rot).view(1, 1, -1)
    cos, sin = torch.cos(angle), torch.sin(angle)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def query_temperature(positions, coef, every):
    return 1.0 + coef * torch.log(torch.floor((positions.to(F64) + 1.0) / every) + 1.0)


def head_slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)


def softmax_with_sink(scores, seen, sink):
    """scores [n, m] of one head, ``seen`` a mask, ``sink`` a number that joins the denominator as exp(sink)."""
    scores = scores.masked_fill(~seen, -math.inf)
    sink = torch.as_tensor(sink, dtype=F64)
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink)
    weights = torch.exp(scores - top)
    return weights / (weights.sum(-1, keepdim=True) + torch.exp(sink - top))


def attend(q, k, v, scale, sinks, slopes=None, temps=None, cap=0.0, offset=0):
    """q [n, H, d] at positions offset.. over k, v [m, G, *] from position 0: scores times ``scale`` (and a number per
    head), capped, lowered by slope * distance, a sink per head.  Returns [n, H, vdim]."""
    n, heads, _ = q.shape
    m, groups, _ = k.shape
    i, j = torch.arange(offset, offset + n).view(-1, 1), torch.arange(m).view(1, -1)
    out = []
    for head in range(heads):
        group = head // (heads // groups)
        s = q[:, head] @ k[:, group].T * scale
        if temps is not None:
            s = s * temps[head]
        if cap:
            s = cap * torch.tanh(s / cap)
        if slopes is not None:
            s = s - slopes[head] * (i - j).to(F64)
        out.append(softmax_with_sink(s, j <= i, sinks[head]) @ v[:, group])
    return torch.stack(out, 1)


def mix_values(v, w, m, carry):
    """Values of the first mixing layer are kept in ``carry``; later ones are blended with them."""
    if not m.get("v_mix"):
        return v
    if "first" not in carry:
        carry["first"] = v
        return v
    lam = w["vmix"]
    return (1.0 - lam) * v + lam * carry["first"]


def biased_mixer(h, w, m, eps, carry):
    """Per-head norm with gains, a temperature that grows with the position, a distance bias, a stored sink and one
    gate a head."""
    tokens, heads, groups = h.shape[0], m["heads"], m["kv_heads"]
    q = rms((h @ w["q"].T).view(tokens, heads, m["dim"]), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).view(tokens, groups, m["dim"]), eps) * w["k.norm"]
    v = mix_values((h @ w["v"].T).view(tokens, groups, m["vdim"]), w, m, carry)
    heat = m["q_temp"]
    q = q * query_temperature(torch.arange(tokens), heat["coef"], heat["every"]).view(-1, 1, 1)
    o = attend(rounded(q), rounded(k), rounded(v), m["scale"], w["sink"], slopes=head_slopes(heads))
    o = o * torch.sigmoid(h @ w["g"].T).unsqueeze(-1)
    return rounded(o.reshape(tokens, -1)) @ w["o"].T


def rotated_mixer(h, w, m, eps, carry):
    """Rotation, then a norm without gains, a number per head on the scores, a soft cap, one in the denominator."""
    tokens, heads, groups = h.shape[0], m["heads"], m["kv_heads"]
    at = torch.arange(tokens)
    q = rms(rotate_pairs((h @ w["q"].T).view(tokens, heads, m["dim"]), at, m["rot"]), eps)
    k = rms(rotate_pairs((h @ w["k"].T).view(tokens, groups, m["dim"]), at, m["rot"]), eps)
    v = mix_values((h @ w["v"].T).view(tokens, groups, m["vdim"]), w, m, carry)
    o = attend(rounded(q), rounded(k), rounded(v), m["scale"], torch.zeros(heads, dtype=F64), temps=w["temp"], cap=m["softcap"])
    return rounded(o.reshape(tokens, -1)) @ w["o"].T


def state_space(x, b, c, dt, a_log, d, state=None):
    """x [T, H, vdim], b and c [T, G, N], dt [T, H] (after softplus): the recurrence token by token.  Returns
    y [T, H, vdim] and the last state [H, N, vdim]."""
    tokens, heads, vdim = x.shape
    groups, n = b.shape[1:]
    of = torch.arange(heads) // (heads // groups)
    state = torch.zeros(heads, n, vdim, dtype=F64) if state is None else state.clone()
    out = []
    for t in range(tokens):
        keep = torch.exp(-torch.exp(a_log) * dt[t])
        bt, ct = b[t, of], c[t, of]
        state = keep.view(-1, 1, 1) * state + dt[t].view(-1, 1, 1) * bt.unsqueeze(-1) * x[t].unsqueeze(-2)
        out.append(torch.einsum("hnv,hn->hv", state, ct) + d.view(-1, 1) * x[t])
    return torch.stack(out), state


def mamba_mixer(h, w, m, eps, carry):
    tokens, heads, vdim, n, groups = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = heads * vdim
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * groups * n, heads], -1)
    xbc = silu(causal_conv(xbc, w["conv"]) + w["conv.b"])
    x, b, c = torch.split(xbc, [inner, groups * n, groups * n], -1)
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
    y, _ = state_space(x.reshape(tokens, heads, vdim), b.reshape(tokens, groups, n), c.reshape(tokens, groups, n), dt,
                       w["A_log"], w["D"])
    y = group_norm(y.reshape(tokens, inner) * silu(z), w["norm"], eps, m["norm_groups"])
    return rounded(y) @ w["o"].T


def choose_experts(h, w, router):
    """Chosen experts [T, top] and their weights."""
    scores = torch.sigmoid(h @ w["router"].T)
    choice = scores + w["correction"]
    experts, count, keep = int(router["experts"]), int(router["groups"]["count"]), int(router["groups"]["keep"])
    by_group = choice.view(-1, count, experts // count)
    strength = torch.topk(by_group, min(2, experts // count), dim=-1).values.sum(-1)
    allowed = torch.zeros_like(strength, dtype=torch.bool).scatter(1, torch.topk(strength, keep, dim=-1).indices, True)
    choice = by_group.masked_fill(~allowed.unsqueeze(-1), -math.inf).reshape(-1, experts)
    ids = torch.topk(choice, int(router["top"]), dim=-1).indices
    share = scores.gather(1, ids)
    return ids, share / (share.sum(-1, keepdim=True) + 1e-20)


def routed_feed_forward(h, w, mlp):
    ids, share = choose_experts(h, w, mlp["router"])
    out = torch.zeros_like(h)
    for expert in range(int(mlp["router"]["experts"])):
        rows, slots = torch.where(ids == expert)
        if rows.numel():
            e = f"e{expert}."
            y = rounded(silu(h[rows] @ w[e + "gate"].T) * (h[rows] @ w[e + "up"].T)) @ w[e + "down"].T
            out[rows] += share[rows, slots].unsqueeze(-1) * y
    return out


def token_side(x, e, w, eps):
    y = rounded(gelu_tanh(rounded(x) @ w["side.gate"].T) * e) @ w["side.proj"].T
    return x + rms(y, eps) * w["side.norm"]


MIXERS = {"mamba2": mamba_mixer, "attention": biased_mixer, "attention_2": rotated_mixer}


def sub(weights, prefix):
    return {name[len(prefix):]: tensor.to(F64) for name, tensor in weights.items() if name.startswith(prefix)}


def read_folder(folder):
    """config.json as a dictionary and the stored tensors by name."""
    import json
    from pathlib import Path

    import safetensors.torch

    with open(Path(folder) / "config.json", encoding="utf-8") as handle:
        config = json.load(handle)
    return config, safetensors.torch.load_file(str(Path(folder) / "model.safetensors"))


def greedy(config, weights, prompt, count):
    """``count`` tokens after ``prompt``, each the argmax (lowest index on ties) of the whole sequence so far."""
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(torch.argmax(forward(config, weights, tokens)[-1])))
    return tokens[len(prompt):]


def forward(config, weights, tokens, streams=None, noise=None):
    """Logits [T, vocab] of one sequence in float64.  ``streams``: a list that receives the stream after every
    layer.  ``noise``: a seed; inputs of products and rows that a cache holds are then each moved by up to the rounding
    of bfloat16, or (0) rounded to it; everything else stays exact."""
    NOISE[0] = None if noise is None else torch.Generator().manual_seed(noise)
    try:
        return _forward(config, weights, tokens, streams)
    finally:
        NOISE[0] = None


def _forward(config, weights, tokens, streams):
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]
    w = {name: tensor.to(F64) for name, tensor in weights.items()}
    ids = torch.as_tensor(tokens, dtype=torch.long)
    side, dim = w["side.embed"][ids], config["token_side"]["dim"]
    x = group_norm(w["embed"][ids], w["embed.norm"], eps, groups)
    carry: dict = {}
    for index, layer in enumerate(config["layers"]):
        lw = sub(w, f"l{index}.")
        h = group_norm(x, lw["norm1"], eps, groups)
        h = rounded(h + causal_conv(h, lw["canon1"]))
        x = x + MIXERS[layer["type"]](h, sub(lw, "mix."), layer["mixer"], eps, carry)
        if layer.get("mlp"):
            x = x + routed_feed_forward(rounded(group_norm(x, lw["norm2"], eps, groups)), sub(lw, "mlp."), layer["mlp"])
        x = token_side(x, side[:, index * dim:(index + 1) * dim], lw, eps)
        if streams is not None:
            streams.append(x)
    return rounded(group_norm(x, w["final.norm"], eps, groups)) @ w["embed"].T * config["logit_scale"]
