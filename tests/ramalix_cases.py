"""Small Ramalix configurations for the tests.  They differ from one another in every size and
option: layer order, which layers repeat and how often, head counts and groups, key, value and
turned sizes, chunks, taps of both convolutions, the experts' groups, the shared expert (wider
than an expert, as wide, narrower, absent), layers without a feed-forward, page sizes."""
from __future__ import annotations

import os

STD = 0.08       # wider than an initialiser's 0.02, so a wrong key, state or gate moves the logits


def attention(heads, kv_heads, dim, vdim, scale, diff, q_temp, mlp):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if kv_heads is not None:
        mixer["kv_heads"] = kv_heads
    if q_temp is not None:
        mixer["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def chunked(heads, kv_heads, dim, vdim, scale, size, rot, base, mlp):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}
    if rot is not None:
        mixer["rot"] = {"base": base, "dims": rot}
    return {"type": "attention_2", "mixer": mixer, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(experts, top, ff, groups=None, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if groups is not None:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def model(vocab, width, eps, mult, logit_scale, taps, layers, loop):
    out = {"architecture": "Ramalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
           "residual_mult": mult, "logit_scale": logit_scale, "layers": layers}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


CASES = {
    # the repeated run is in the middle and holds all three mixers; a layer without a feed-forward
    "ra-a": dict(seed=3, page_tokens=16, config=model(300, 64, 1e-6, 0.7, 1.5, 4, [
        delta(4, 2, 16, 24, 4, moe(6, 2, 24, (3, 2), 40)),
        attention(4, 2, 16, 24, 0.5, 0.3, (0.2, 10), moe(8, 3, 16, (4, 2), 16)),
        chunked(4, 2, 16, 24, 0.5, 21, 8, 1000.0, None),
        delta(2, 2, 24, 8, 3, moe(5, 2, 20, None, 8)),
        chunked(2, 1, 32, 32, 0.4, 40, 32, 500.0, moe(4, 1, 32, (2, 1), None))], (1, 4, 2))),
    # the repeated run starts at the first layer and runs three times; sizes that are no
    # multiples of 8; one key/value head; no rotation and no temperature on some layers
    "ra-b": dict(seed=4, page_tokens=8, config=model(211, 44, 1e-5, 1.3, 0.6, 2, [
        chunked(3, 1, 10, 14, 0.6, 7, None, 1.0, moe(3, 3, 12, None, 30)),
        delta(6, 3, 10, 6, 2, None),
        attention(3, 1, 12, 20, 0.6, 0.8, None, moe(6, 2, 10, (2, 1), 10)),
        chunked(5, 5, 4, 6, 0.7, 64, 2, 50.0, moe(9, 4, 7, (3, 3), 20))], (0, 2, 3))),
    # sizes that let the bfloat16 products and attentions run on the tensor cores; the repeated
    # run is the last layer alone
    "ra-c": dict(seed=5, page_tokens=16, config=model(400, 128, 1e-5, 0.4, 2.5, 3, [
        chunked(4, 2, 64, 64, 0.1, 50, 48, 9000.0, moe(8, 2, 64, (4, 2), 128)),
        attention(4, 2, 32, 64, 0.12, 0.5, (0.4, 16), moe(4, 2, 72, (2, 2), 72)),
        delta(4, 1, 64, 32, 4, moe(8, 4, 40, (2, 1), 64)),
        attention(2, 2, 64, 128, 0.08, 0.2, (0.1, 100), moe(4, 3, 64, None, 24)),
        chunked(8, 2, 128, 128, 0.05, 96, 64, 9000.0, moe(4, 1, 64, None, None))], (4, 5, 2))),
    # no repeated run at all; one tap in both convolutions; keys and values of unlike
    # tensor-core sizes; a chunk longer than any request
    "ra-d": dict(seed=6, page_tokens=32, config=model(150, 48, 1e-6, 1.0, 1.0, 1, [
        attention(6, 3, 8, 48, 0.9, 0.6, (0.5, 3), None),
        delta(1, 1, 40, 12, 1, moe(2, 1, 64, (1, 1), 64)),
        chunked(4, 1, 48, 16, 0.5, 4000, 16, 77.0, moe(4, 2, 8, (4, 2), 8)),
        attention(2, 1, 24, 16, 0.4, 0.9, None, moe(4, 2, 8, (2, 1), 8))], None)),
}


SIGNS = 3        # features of the residual that only the embedding writes, for `decisive_routers`


def decisive_routers(config):
    """An edit of a model's tensors after which no token's choice of experts is a close call, so
    that bfloat16 chooses what the plain model does: the residual's first features hold one of
    eight sign patterns, given by the token and written by nothing else; the routers read little
    beside them, by matrices drawn until every pattern's choice is clear by a wide margin."""
    import itertools

    import torch

    def edit(t):
        g = torch.Generator().manual_seed(12)
        n = SIGNS
        t["embed"][:, :n] = (0.2 * (torch.randint(0, 2, (t["embed"].shape[0], n), generator=g) * 2 - 1)).to(torch.bfloat16)
        if "loop.step" in t:
            t["loop.step"][:, :n] = 0
        for name in t:
            if name.split(".")[-1] in ("o", "down") or name.endswith(".o.b"):
                t[name][:n] = 0
            elif name.endswith("canon1") or name.endswith("canon2"):
                t[name][:n] = 0
        patterns = torch.tensor(list(itertools.product([-1.0, 1.0], repeat=n)))
        for i, layer in enumerate(config["layers"]):
            if layer.get("mlp") is None:
                continue
            r = layer["mlp"]["router"]
            groups = r.get("groups") or {"count": 1, "keep": 1}
            best, best_margin = None, -1.0
            for _ in range(400):
                m = torch.randn(r["experts"], n, generator=g)
                margin = min(_margin((m @ p).tolist(), r["top"], groups["count"], groups["keep"]) for p in patterns)
                if margin > best_margin:
                    best, best_margin = m, margin
            w = t[f"l{i}.mlp.router"].float() * 0.02
            w[:, :n] = best * 2.0
            t[f"l{i}.mlp.router"] = w.to(torch.bfloat16)
    return edit


def _margin(z, top, groups, keep):
    """How far the choice is from another one: the gap behind the last kept group and the one
    behind the last chosen expert."""
    size = len(z) // groups
    best = sorted(((max(z[g * size:(g + 1) * size]), g) for g in range(groups)), reverse=True)
    gap = best[keep - 1][0] - best[keep][0] if keep < groups else 9.0
    kept = {g for _, g in best[:keep]}
    order = sorted((z[e] for e in range(len(z)) if e // size in kept), reverse=True)
    return min(gap, order[top - 1] - order[top] if top < len(order) else 9.0)


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
