"""A plain, slow restatement of the Ramalix design in PyTorch on the CPU, one function per
mechanism, written from the design's equations and sharing no code with the engine.  Whole
sequences only: no cache and no state handed between calls; every key is recomputed and every
recurrence and convolution starts at zero.  `dtype` is the arithmetic type (float64 for an oracle).

Notation: T tokens, W model width, H query (or value) heads, G key/value (or query/key) heads;
weights are [out, in] and applied as x @ w.T; positions count from 0.  A layer is
    x <- x + m mixer(conv(n1)),  x <- x + m ff(conv(n2)),
n = unit_rms(x) * g with ONE number g, conv(n)_t = n_t + a causal convolution of n per channel.
A run of layers may repeat: before every pass but the first the embedding's output is added to
x, before every pass a learned vector is.
"""
from __future__ import annotations

import json
import math
import os

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def norm_one_number(x, g, eps):
    """One number is the gain of every coordinate."""
    return unit_rms(x, eps) * g


def causal_conv(x, taps_weight):
    """x [T, C], taps_weight [C, taps]; the last column meets the current token, zeros before
    the sequence."""
    t, taps = x.shape[0], taps_weight.shape[1]
    out = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < t:
            out[back:] += x[:t - back] * taps_weight[:, j]
    return out


def input_conv(h, taps_weight):
    return h + causal_conv(h, taps_weight)


def turn_neighbours(x, positions, dims, base):
    """x [T, heads, n]: of the first `dims` features, feature 2i pairs with 2i + 1."""
    if not dims:
        return x
    i = torch.arange(dims // 2, dtype=x.dtype)
    a = positions.to(x.dtype)[:, None] * (base ** (-2.0 * i / dims))[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., dims:]], -1)


def softmax_over(scores, seen, sink=None):
    """scores [H, T, T], seen [T, T] bool.  `sink` [H]: exp(sink) joins every row's denominator
    once, unscaled, with no value."""
    scores = scores.masked_fill(~seen, -math.inf)
    top = scores.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(scores - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink[:, None, None] - top)
    return e / total


def seen_causal(t):
    return torch.ones(t, t, dtype=torch.bool).tril()


def seen_in_chunk(t, size):
    """Row i sees j <= i of its own chunk of `size` positions."""
    chunk = torch.arange(t) // size
    return seen_causal(t) & (chunk[:, None] == chunk[None, :])


def query_temperature(positions, coef, every, dtype):
    return 1.0 + coef * torch.log(((positions + 1) // every).to(dtype) + 1.0)


# ---- mixers ---------------------------------------------------------------------------------

def differential_attention(h, w, m, eps, prefix):
    """Two softmax maps per head over the same values; a1 - lambda a2, unit rms over the head's
    values, times 1 - diff.  Biases on every projection, no rotation, queries that grow with the
    logarithm of their position."""
    t = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, E = m.get("kv_heads", H), m.get("vdim", D)
    q = (h @ w[prefix + "q"].T + w[prefix + "q.b"]).view(t, H, 2, D)
    k = (h @ w[prefix + "k"].T + w[prefix + "k.b"]).view(t, G, 2, D).repeat_interleave(H // G, dim=1)
    v = (h @ w[prefix + "v"].T + w[prefix + "v.b"]).view(t, G, E).repeat_interleave(H // G, dim=1)
    if m.get("q_temp"):
        q = q * query_temperature(torch.arange(t), m["q_temp"]["coef"], m["q_temp"]["every"], h.dtype)[:, None, None, None]
    maps = []
    for i in range(2):
        p = softmax_over(torch.einsum("ihd,jhd->hij", q[:, :, i], k[:, :, i]) * m["scale"], seen_causal(t))
        maps.append(torch.einsum("hij,jhe->ihe", p, v))
    lam = (torch.exp((w[prefix + "lq1"] * w[prefix + "lk1"]).sum())
           - torch.exp((w[prefix + "lq2"] * w[prefix + "lk2"]).sum()) + m["diff"])
    o = unit_rms(maps[0] - lam * maps[1], eps) * (1.0 - m["diff"])
    return o.reshape(t, H * E) @ w[prefix + "o"].T + w[prefix + "o.b"]


def chunked_attention(h, w, m, eps, prefix):
    """Grouped queries, neighbouring pairs turned, keys of the row's own chunk alone, a sink."""
    t = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, E = m.get("kv_heads", H), m.get("vdim", D)
    pos = torch.arange(t)
    q = (h @ w[prefix + "q"].T).view(t, H, D)
    k = (h @ w[prefix + "k"].T).view(t, G, D)
    v = (h @ w[prefix + "v"].T).view(t, G, E)
    rot = m.get("rot")
    if rot:
        q = turn_neighbours(q, pos, rot["dims"], rot["base"])
        k = turn_neighbours(k, pos, rot["dims"], rot["base"])
    k = k.repeat_interleave(H // G, dim=1)
    v = v.repeat_interleave(H // G, dim=1)
    seen = seen_in_chunk(t, m["mask"]["size"]) if m.get("mask") else seen_causal(t)
    p = softmax_over(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], seen, w[prefix + "sink"])
    return torch.einsum("hij,jhe->ihe", p, v).reshape(t, H * E) @ w[prefix + "o"].T


def channel_delta(h, w, m, eps, prefix, states=None):
    """The delta rule with a decay per key channel.  `states`: a list that receives the state
    after the last token."""
    t = h.shape[0]
    H, G, D = m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    E = m.get("vdim", D)

    def through(name):
        return silu(causal_conv(h @ w[prefix + name].T, w[prefix + name + ".conv"]))

    def unit(x):
        return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q = (unit(through("q").view(t, G, D)) * D ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(through("k").view(t, G, D)).repeat_interleave(H // G, dim=1)
    v = through("v").view(t, H, E)
    beta = sigmoid(h @ w[prefix + "b"].T)
    rate = softplus((h @ w[prefix + "a1"].T) @ w[prefix + "a2"].T + w[prefix + "dt_bias"]).view(t, H, D)
    decay = torch.exp(-torch.exp(w[prefix + "A_log"])[None, :, None] * rate)
    S = torch.zeros(H, D, E, dtype=h.dtype)
    o = torch.zeros(t, H, E, dtype=h.dtype)
    for i in range(t):
        S = decay[i][:, :, None] * S
        u = beta[i][:, None] * (v[i] - torch.einsum("hde,hd->he", S, k[i]))
        S = S + k[i][:, :, None] * u[:, None, :]
        o[i] = torch.einsum("hde,hd->he", S, q[i])
    if states is not None:
        states.append(S)
    gate = sigmoid((h @ w[prefix + "g1"].T) @ w[prefix + "g2"].T).view(t, H, E)
    o = unit_rms(o, eps) * w[prefix + "norm"] * gate
    return o.reshape(t, H * E) @ w[prefix + "o"].T


MIXERS = {"attention": differential_attention, "attention_2": chunked_attention, "channel_delta": channel_delta}


# ---- feed-forward -----------------------------------------------------------------------------

def gated(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def choose_experts(s, top, groups, keep):
    """s [E] scores -> the chosen experts' indices: of the `groups` equal runs of neighbours only
    the `keep` with the largest best score take part."""
    size = s.shape[0] // groups
    best = [(-float(s[g * size:(g + 1) * size].max()), g) for g in range(groups)]
    kept = {g for _, g in sorted(best)[:keep]}
    order = sorted((-float(s[e]), e) for e in range(s.shape[0]) if e // size in kept)
    return [e for _, e in order[:top]]


def mixture(h, w, mlp, prefix):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(h @ w[prefix + "router"].T, -1)
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        chosen = choose_experts(s[i], r["top"], groups["count"], groups["keep"])
        total = sum(s[i, e] for e in chosen) + 1e-20
        for e in chosen:
            out[i] += s[i, e] / total * gated(h[i:i + 1], w, f"{prefix}e{e}.")[0]
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[prefix + "shared.sg"].T) * gated(h, w, prefix + "shared.")
    return out


# ---- the model ------------------------------------------------------------------------------

def run_list(config):
    """[(layer, number of the pass or None, first of its pass)]."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, None, False) for i in range(start)]
    for t in range(times):
        out += [(i, t, i == start) for i in range(start, stop)]
    return out + [(i, None, False) for i in range(stop, n)]


def forward(config, w, tokens, dtype=torch.float64, residuals=None):
    """Logits [T, vocab] of one whole sequence.  `residuals`: a list that receives x after
    every layer run."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = embedded = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, number, first in run_list(config):
        layer = config["layers"][i]
        if first:
            if number > 0:
                x = x + embedded
            x = x + w["loop.step"][number]
        h = input_conv(norm_one_number(x, w[f"l{i}.norm1"], eps), w[f"l{i}.canon1"])
        x = x + m * MIXERS[layer["type"]](h, w, layer["mixer"], eps, f"l{i}.mix.")
        if layer.get("mlp") is not None:
            h = input_conv(norm_one_number(x, w[f"l{i}.norm2"], eps), w[f"l{i}.canon2"])
            x = x + m * mixture(h, w, layer["mlp"], f"l{i}.mlp.")
        if residuals is not None:
            residuals.append(x.clone())
    return (norm_one_number(x, w["final.norm"], eps) @ w["head"].T) * config["logit_scale"]


def load_folder(path):
    """(config, tensors) of a model folder; reads the safetensors container itself."""
    import numpy as np
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        n = int.from_bytes(f.read(8), "little")
        header = json.loads(f.read(n))
        data = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = np.frombuffer(data[lo:hi], dtype=np.uint8).copy()
        out[name] = torch.from_numpy(raw).view(kinds[meta["dtype"]]).reshape(meta["shape"])
    return config, out


def greedy(config, w, prompt, n, dtype=torch.float64):
    """`n` tokens after `prompt`, each the largest logit (the lowest index on ties); the whole
    sequence is run again for every token."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(torch.argmax(forward(config, w, tokens, dtype)[-1])))
    return tokens[len(prompt):]
