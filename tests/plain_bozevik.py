"""Bozevik in plain double-precision PyTorch: one function per mechanism, whole sequences only, no cache.

The oracle of the Bozevik tests.  It shares nothing with the product path: it takes the configuration as the
dictionary that config.json holds and the weights as a dictionary of tensors by their stored names, and walks
a whole sequence at once, so every cutting of a prompt, every batch and every page layout of the engine is held
to the same numbers.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def centred_norm(x, gain, eps):
    """Layer norm with a gain and no bias."""
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * gain


def rms_norm(x, gain, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def shifted(x, share):
    """Every row moved towards the row before it by ``share`` per element (the first towards zeros)."""
    before = torch.cat([torch.zeros_like(x[:1]), x[:-1]])
    return x + (before - x) * share


def depth_average(states, share):
    """sum_j share[j] * states[j] over everything the layers have left so far, the embedding rows first."""
    assert len(states) == share.numel()
    return sum(weight * state for weight, state in zip(share, states))


def rotate_pairs(x, positions, base):
    """x: [T, heads, size], all of it turned: elements 2i and 2i + 1 by position * base^(-2i / size)."""
    size = x.shape[-1]
    freq = torch.tensor([float(base) ** (-2.0 * i / size) for i in range(size // 2)], dtype=F64)
    angle = positions.to(F64).view(-1, 1, 1) * freq.view(1, 1, -1)
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * torch.cos(angle) - v * torch.sin(angle)
    out[..., 1::2] = v * torch.cos(angle) + u * torch.sin(angle)
    return out


def cached_rows(h, w, m, eps):
    """What a layer with a down projection leaves for itself and for layers that read it: (latents [T, rank], turned
    key parts [T, rot_dim])."""
    rank = m["kv_rank"]
    down = h @ w["dkv"].T
    turned = rotate_pairs(down[:, rank:].unsqueeze(1), torch.arange(h.shape[0]), m["rot"]["base"])[:, 0]
    return rms_norm(down[:, :rank], w["dkv.norm"], eps), turned


def latent_attention(h, w, m, eps, latent, k_turned):
    heads, dim, rot_dim, vdim = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    tokens = h.shape[0]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(tokens, heads, dim + rot_dim)
    q_plain, q_turned = q[..., :dim], rotate_pairs(q[..., dim:], torch.arange(tokens), m["rot"]["base"])
    k_plain = (latent @ w["uk"].T).view(tokens, heads, dim)
    values = (latent @ w["uv"].T).view(tokens, heads, vdim)
    later = torch.triu(torch.ones(tokens, tokens, dtype=torch.bool), diagonal=1)
    out = []
    for head in range(heads):
        scores = (q_plain[:, head] @ k_plain[:, head].T + q_turned[:, head] @ k_turned.T) * m["scale"]
        out.append(torch.softmax(scores.masked_fill(later, -math.inf), -1) @ values[:, head])
    return torch.cat(out, -1) @ w["o"].T


def clamped_unit(h, w, limit):
    g = torch.clamp(h @ w["gate"].T, max=limit)
    u = torch.clamp(h @ w["up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def routed_units(h, w, mlp):
    """Each token's best experts see the token's row times their own score; a shared unit sees the row itself."""
    scores = torch.sigmoid(h @ w["router"].T)
    best = torch.topk(scores, int(mlp["router"]["top"]), dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for score, expert in zip(best.values[t], best.indices[t].tolist()):
            out[t] += clamped_unit(score * h[t], sub(w, f"e{expert}."), mlp["expert"]["limit"])
    if mlp.get("shared"):
        out = out + clamped_unit(h, sub(w, "shared."), mlp["shared"]["limit"])
    return out


def sub(weights, prefix):
    return {name[len(prefix):]: tensor.to(F64) for name, tensor in weights.items() if name.startswith(prefix)}


def rounded(h, on):
    """The sublayer's input as a bfloat16 product would see it (``on``), or as it is."""
    return h.to(torch.bfloat16).to(F64) if on else h


def run_layer(x, config, weights, index, kept, round_inputs=False):
    """One layer on the stream of a whole sequence; ``kept``: cached rows by layer (grows)."""
    layer, eps = config["layers"][index], config["norm"]["eps"]
    w, m = sub(weights, f"l{index}."), layer["mixer"]
    mix = sub(w, "mix.")
    h = rounded(shifted(x, w["shift"]), round_inputs)
    source = m.get("kv_from")
    if source is None:
        kept[index] = cached_rows(h, mix, m, eps)
        source = index
    x = x + centred_norm(latent_attention(h, mix, m, eps, *kept[source]), w["norm1"], eps)
    mlp = layer.get("mlp")
    if mlp:
        h, ff = rounded(x, round_inputs), sub(w, "mlp.")
        y = clamped_unit(h, ff, mlp["limit"]) if mlp["kind"] == "dense" else routed_units(h, ff, mlp)
        x = x + centred_norm(y, w["norm2"], eps)
    return x


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


def forward(config, weights, tokens, streams=None, round_inputs=False):
    """Logits [T, vocab] of one sequence in float64.  ``streams``: a list that receives the stream after every layer,
    averaged over depth.  ``round_inputs``: every sublayer reads its input rounded to bfloat16 (everything else stays
    exact)."""
    w = {name: tensor.to(F64) for name, tensor in weights.items()}
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    states, kept = [x], {}
    for index in range(len(config["layers"])):
        states.append(run_layer(x, config, weights, index, kept, round_inputs))
        x = depth_average(states, w[f"l{index}.dwa"])
        if streams is not None:
            streams.append(x)
    x = centred_norm(x, w["final.norm"], config["norm"]["eps"])
    return x @ w["embed"].T * config["logit_scale"]
