"""A plain, slow restatement of the Gavipel design in PyTorch on the CPU, one function per
mechanism, written from the design's equations and sharing no code with the engine.  Whole
sequences only: no cache handed between calls, every key is recomputed.  `dtype` is the arithmetic
type (float64 for an oracle).

Notation: T tokens, W model width, H query heads, G key/value heads; weights are [out, in] and
applied as x @ w.T; positions count from 0.  A layer is
    x <- x + (s1 * mixer(n1(x)) + s2 * ff(n2(x))),
both norms of the same x, s1 and s2 vectors over W.  A run of layers may repeat: x passes one matrix
product together with the embedding's output before every pass.
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


def norm_around_one(x, w, eps):
    """The weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def head_norm(x, w, eps):
    """x [T, heads, n]; one plain weight over n for all heads."""
    return unit_rms(x, eps) * w


def turning_rates(dims, base, scaling=None):
    """Radians a position of every pair of the first `dims` features.  `scaling` = {factor, low,
    high, original}: wavelengths over original / low slow down by the factor, those under
    original / high stay, those between go over linearly in original / wavelength."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            length = 2.0 * math.pi / f
            if length > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif not length < scaling["original"] / scaling["high"]:
                s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def turn_neighbours(x, positions, dims, base, scaling=None):
    """x [T, heads, n]: of the first `dims` features, feature 2i pairs with 2i + 1."""
    if not dims:
        return x
    a = (positions.to(torch.float64)[:, None] * turning_rates(dims, base, scaling)[None, :]).to(x.dtype)
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., dims:]], -1)


def seen_in_window(t, size=None):
    """Row i sees j with 0 <= i - j < size; every earlier key without a size."""
    back = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return (back >= 0) & (back < (size if size is not None else t + 1))


def softmax_plus_one(scores, seen):
    """exp(s) / (1 + sum exp(s)) over the seen keys."""
    scores = scores.masked_fill(~seen, -math.inf)
    top = torch.clamp(scores.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


# ---- the mixer --------------------------------------------------------------------------------

def attention(h, w, m, eps, prefix):
    t = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, E = m.get("kv_heads", H), m.get("vdim", D)
    pos = torch.arange(t)
    q = head_norm((h @ w[prefix + "q"].T).view(t, H, D), w[prefix + "q.norm"], eps)
    k = head_norm((h @ w[prefix + "k"].T).view(t, G, D), w[prefix + "k.norm"], eps)
    v = (h @ w[prefix + "v"].T).view(t, G, E)
    rot = m.get("rot")
    if rot:
        q = turn_neighbours(q, pos, rot["dims"], rot["base"], rot.get("scaling"))
        k = turn_neighbours(k, pos, rot["dims"], rot["base"], rot.get("scaling"))
    seen = seen_in_window(t, m["mask"]["size"] if m.get("mask") else None)
    out = []
    for i in range(H):
        g = i // (H // G)
        p = softmax_plus_one((q[:, i] @ k[:, g].T) * m["scale"], seen)
        out.append(p @ v[:, g])
    o = torch.cat(out, -1) * sigmoid(h @ w[prefix + "g"].T)
    return o @ w[prefix + "o"].T


# ---- the feed-forward ---------------------------------------------------------------------------

def gated(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def choose_experts(choice, top, groups, keep):
    """choice [E] -> the chosen experts' indices: of the `groups` equal runs of neighbours only the
    `keep` whose two largest choice scores have the largest sum take part."""
    size = choice.shape[0] // groups
    sums = []
    for g in range(groups):
        best = sorted((float(c) for c in choice[g * size:(g + 1) * size]), reverse=True)[:2]
        sums.append((-sum(best), g))
    kept = {g for _, g in sorted(sums)[:keep]}
    order = sorted((-float(choice[e]), e) for e in range(choice.shape[0]) if e // size in kept)
    return [e for _, e in order[:top]]


def mixture(h, w, mlp, prefix):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = sigmoid(h @ w[prefix + "router"].T)
    choice = s + w[prefix + "correction"]
    weight = torch.zeros_like(s)
    for i in range(h.shape[0]):
        for e in choose_experts(choice[i], r["top"], groups["count"], groups["keep"]):
            weight[i, e] = s[i, e]
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows = weight[:, e].nonzero().flatten()
        if len(rows):
            out[rows] += weight[rows, e:e + 1] * gated(h[rows], w, f"{prefix}e{e}.")
    if mlp.get("shared"):
        out = out + gated(h, w, prefix + "shared.")
    return out


# ---- the model ------------------------------------------------------------------------------

def run_list(config):
    """[(layer, first of a pass)]."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, False) for i in range(start)]
    for _ in range(times):
        out += [(i, i == start) for i in range(start, stop)]
    return out + [(i, False) for i in range(stop, n)]


def enter_pass(x, embedded, w_in):
    return torch.cat([x, embedded], -1) @ w_in.T


def forward(config, w, tokens, dtype=torch.float64, residuals=None):
    """Logits [T, vocab] of one whole sequence.  `residuals`: a list that receives x after
    every layer run."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = config["norm"]["eps"]
    x = embedded = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for i, first in run_list(config):
        layer = config["layers"][i]
        if first:
            x = enter_pass(x, embedded, w["loop.in"])
        add = w[f"l{i}.ls1"] * attention(norm_around_one(x, w[f"l{i}.norm1"], eps), w, layer["mixer"], eps, f"l{i}.mix.")
        if layer.get("mlp") is not None:
            add = add + w[f"l{i}.ls2"] * mixture(norm_around_one(x, w[f"l{i}.norm2"], eps), w, layer["mlp"], f"l{i}.mlp.")
        x = x + add
        if residuals is not None:
            residuals.append(x.clone())
    return norm_around_one(x, w["final.norm"], eps) @ w["embed"].T


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
