"""Small Gavipel configurations for the tests.  They differ from one another in every size and
option: which layers repeat and how often, head counts and groups, key, value and turned sizes,
windows (absent too), the rotation's stretching (absent too), the experts' groups, the shared expert
(wider than an expert, as wide, narrower, absent), layers without a feed-forward, page sizes."""
from __future__ import annotations

import itertools
import os

import torch

STD = 0.08       # wider than an initialiser's 0.02, so a wrong key or gate moves the logits


def attention(heads, kv_heads, dim, vdim, scale, window, rot, mlp):
    """rot: None or (dims, base) or (dims, base, (factor, low, high, original))."""
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "scale": scale}
    if kv_heads is not None:
        mixer["kv_heads"] = kv_heads
    if window is not None:
        mixer["mask"] = {"size": window}
    if rot is not None:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            mixer["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), rot[2]))
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def moe(experts, top, ff, groups=None, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if groups is not None:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, eps, scale, layers, loop):
    out = {"architecture": "Gavipel", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": scale}, "layers": layers}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


CASES = {
    # the repeated run is in the middle; a layer without a feed-forward in it
    "ga-a": dict(seed=3, page_tokens=16, config=model(300, 64, 1e-6, 7.3, [
        attention(4, 2, 16, 24, 0.4, 21, (8, 1000.0, (8.0, 1.0, 3.0, 40.0)), moe(6, 2, 24, (3, 2), 40)),
        attention(4, 1, 16, 16, 0.5, 40, (16, 1000.0), moe(8, 3, 16, (4, 2), 16)),
        attention(6, 3, 24, 8, 0.3, None, (12, 300.0, (3.0, 0.5, 2.0, 100.0)), None),
        attention(2, 2, 32, 32, 0.25, 9, None, moe(5, 2, 20, None, 8)),
        attention(4, 2, 16, 24, 0.4, 21, (8, 1000.0, (8.0, 1.0, 3.0, 40.0)), moe(4, 1, 32, (2, 1), None))], (1, 4, 2))),
    # the repeated run starts at the first layer and runs three times; sizes that are no multiples
    # of 8, odd ones among them; a window of two tokens
    "ga-b": dict(seed=4, page_tokens=8, config=model(211, 44, 1e-5, 3.0, [
        attention(3, 1, 10, 14, 0.6, 2, (4, 50.0), moe(3, 3, 12, None, 30)),
        attention(5, 5, 6, 9, 0.7, 64, (2, 50.0, (2.0, 1.0, 2.0, 10.0)), moe(9, 4, 7, (3, 3), 20)),
        attention(2, 1, 15, 7, 0.4, 33, (14, 500.0), None),
        attention(6, 2, 12, 20, 0.6, None, None, moe(6, 2, 10, (6, 2), 10))], (0, 2, 3))),
    # sizes that let the bfloat16 products and attentions run on the tensor cores; the repeated run
    # is the last layer alone
    "ga-c": dict(seed=5, page_tokens=16, config=model(400, 128, 1e-5, 11.0, [
        attention(4, 2, 64, 64, 0.125, 50, (48, 9000.0, (4.0, 1.0, 4.0, 256.0)), moe(8, 2, 64, (4, 2), 128)),
        attention(8, 2, 128, 128, 0.09, 96, (64, 9000.0), moe(16, 4, 40, (4, 3), 72)),
        attention(4, 1, 48, 80, 0.15, 70, (48, 400.0, (4.0, 1.0, 4.0, 256.0)), moe(4, 2, 72, (2, 2), None)),
        attention(2, 2, 128, 128, 0.09, 40, (128, 9000.0, (16.0, 2.0, 8.0, 64.0)), moe(8, 4, 64, (2, 1), 24))], (3, 4, 2))),
    # no repeated run; one key/value head; a window longer than any request
    "ga-d": dict(seed=6, page_tokens=32, config=model(150, 48, 1e-6, 1.0, [
        attention(6, 3, 8, 48, 0.9, 4000, (8, 77.0), None),
        attention(4, 1, 48, 16, 0.3, 17, (16, 77.0, (5.0, 1.0, 1.0, 20.0)), moe(4, 2, 8, (4, 2), 8)),
        attention(2, 1, 24, 16, 0.4, None, (24, 10.0), moe(2, 1, 64, (1, 1), 64))], None)),
}


SIGNS = 3        # features of the residual that only the embedding writes, for `decisive_routers`


def margin(choice, top, groups, keep):
    """How far a choice of experts is from another one: the gap behind the last kept group's sum of
    two, and the one behind the last chosen expert."""
    size = len(choice) // groups
    sums = sorted((sum(sorted(choice[g * size:(g + 1) * size], reverse=True)[:2]), g) for g in range(groups))[::-1]
    gap = sums[keep - 1][0] - sums[keep][0] if keep < groups else 9.0
    kept = {g for _, g in sums[:keep]}
    order = sorted((choice[e] for e in range(len(choice)) if e // size in kept), reverse=True)
    return min(gap, order[top - 1] - order[top] if top < len(order) else 9.0)


def decisive_routers(config):
    """An edit of a model's tensors after which no token's choice of experts is a close call, so
    that bfloat16 chooses what the plain model does: the residual's first features hold one of eight
    sign patterns, given by the token and written by nothing else; the routers read little beside
    them, by matrices and corrections drawn until every pattern's choice is clear at any size the
    norm may leave the pattern."""
    def edit(t):
        g = torch.Generator().manual_seed(12)
        n = SIGNS
        t["embed"][:, :n] = (0.4 * (torch.randint(0, 2, (t["embed"].shape[0], n), generator=g) * 2 - 1)).to(torch.bfloat16)
        if "loop.in" in t:
            t["loop.in"][:n] = 0
            for i in range(n):
                t["loop.in"][i, i] = 1.0
        for name in t:
            if name.split(".")[-1] in ("o", "down"):
                t[name][:n] = 0
            elif name.endswith("norm2"):
                t[name][:n] = 0
        patterns = torch.tensor(list(itertools.product([-1.0, 1.0], repeat=n)))
        for i, layer in enumerate(config["layers"]):
            if layer.get("mlp") is None:
                continue
            r = layer["mlp"]["router"]
            groups = r.get("groups") or {"count": 1, "keep": 1}
            # of the draws that are clear enough, the one that tells the patterns apart best
            best, best_rank = None, (-1, -1.0)
            for _ in range(400):
                m = 1.5 * torch.randn(r["experts"], n, generator=g)
                c = 0.3 * torch.randn(r["experts"], generator=g) - 0.5
                scores = [[(torch.sigmoid(size * (m @ p)) + c).tolist() for size in (1.0, 1.5, 2.0, 2.5, 3.0)] for p in patterns]
                worst = min(margin(z, r["top"], groups["count"], groups["keep"]) for row in scores for z in row)
                kinds = len({tuple(sorted(range(r["experts"]), key=lambda e: -row[1][e])[:r["top"]]) for row in scores})
                rank = (kinds if worst > 0.08 else 0, worst)
                if rank > best_rank:
                    best, best_rank = (m, c), rank
            w = t[f"l{i}.mlp.router"].float() * 0.01
            w[:, :n] = best[0]
            t[f"l{i}.mlp.router"] = w.to(torch.bfloat16)
            t[f"l{i}.mlp.correction"] = best[1].to(t[f"l{i}.mlp.correction"].dtype)
    return edit


def make_folder(tmp_path, name, config=None, seed=None, edit=None) -> str:
    """`edit`: a function of the dict of tensors, applied before they are written (default: routers
    whose choices are clear)."""
    from crucible_b200.weights import write_random_model
    out = os.path.join(str(tmp_path), name)
    case = CASES.get(name, {})
    write_random_model(config or case["config"], out, case.get("seed", 0) if seed is None else seed, std=STD)
    if edit is None:
        edit = decisive_routers(config or case["config"])
    if edit:
        from crucible_b200.weights.safetensors_io import SafetensorsFile, write_safetensors
        path = os.path.join(out, "model.safetensors")
        f = SafetensorsFile(path)
        tensors = {n: f.get(n) for n in f.names()}
        f.close()
        edit(tensors)
        write_safetensors(path, tensors)
    return out
