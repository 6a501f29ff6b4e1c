"""Each mechanism of the Gavipel design alone: its part, driven over hand-made steps, against the
one-mechanism functions of `plain_gavipel.py`.  Inputs are made so that a fault shows: marked keys
whose scores stand out at window and page borders, softmaxes whose sink takes most of the weight,
experts whose choice scores are all negative, groups whose best expert and best two disagree."""
import pytest
import torch

import plain_gavipel as plain
from test_futepel_kernels_gpu import DEV, TOL, Steps, _bind, _i32, rel
from test_nipapel_kernels_gpu import StepsWithValues, _cuts, _run_part

pytestmark = pytest.mark.gpu


# ---------------------------------------------------------------------------
# windowed attention: head norms, neighbouring pairs with stretched rates, a fixed sink, a gate
# ---------------------------------------------------------------------------

SCALING = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 90.0}


def _spec(H, G, D, E, R, window, width, scale, scaling=SCALING):
    from crucible_b200.config.model_config import MixerSpec, PositionSpec
    position = PositionSpec("rope_interleaved", R, 700.0, 0, tuple(scaling.items()) if scaling else None) if R else None
    return MixerSpec(kind="sink_attention", width=width, n_heads=H, n_kv_heads=G, head_dim=D, softmax_scale=scale,
                     window=window, position=position,
                     extra=(("value_dim", E), ("keep_first", 0), ("sink", 0.0), ("gate", "element"),
                            ("value_norm_eps", None), ("qk_norm_eps", 1e-5)))


def _cfg(H, G, D, E, R, window, scale, scaling=SCALING):
    out = {"heads": H, "kv_heads": G, "dim": D, "vdim": E, "scale": scale}
    if R:
        out["rot"] = {"dims": R, "base": 700.0, "scaling": scaling}
    if window:
        out["mask"] = {"size": window}
    return out


KINDS = [
    (torch.float32, 16, 24, False), (torch.float32, 15, 9, False), (torch.bfloat16, 20, 12, False),
    (torch.bfloat16, 32, 32, False), (torch.bfloat16, 32, 32, True), (torch.bfloat16, 48, 16, True),
    (torch.bfloat16, 80, 80, True), (torch.bfloat16, 16, 80, True),
    # heads of 64 and 128: portions of 32 tokens and more on the tcgen05 tiles
    (torch.bfloat16, 64, 64, True), (torch.bfloat16, 128, 128, True)]


@pytest.mark.parametrize("dtype,D,E,tensor_cores", KINDS)
@pytest.mark.parametrize("how", ["prompt", "portions", "decode"])
@pytest.mark.parametrize("window,T", [(10, 90), (70, 300), (1, 20), (64, 140), (500, 120), (None, 150)])
def test_attention_sees_exactly_its_keys(dtype, D, E, tensor_cores, how, window, T, monkeypatch):
    """Feature 0 of the input is 1 for every token and feature 1 for a few marked ones; a channel that
    is not turned reads feature 0 in every query head and feature 1 in every key head, with weights so
    large that it is all the head's norm leaves: a row is held by the marked keys that it may see, and
    by the sink where it sees none."""
    from crucible_b200.ops import sink_attention as k
    from crucible_b200.parts import MIXERS, LayerBinding
    monkeypatch.setattr(k, "TENSOR_CORES", tensor_cores)
    H, G, R, width, page, scale = 4, 2, 8, 48, 8, 6.0 / D       # a marked key's score is about D * scale
    marked = sorted(j for j in {0, 7, 8, 40, 63, 64, 130} if j < T - 1)

    def edit(t):
        for name, heads, feature in (("q", H, 0), ("k", G, 1)):
            m = t[name].view(heads, D, width)
            m[:, :, feature] = 0.0
            m[:, D - 1, :] = 0.0
            m[:, D - 1, feature] = 40.0
            t[name + ".norm"] = torch.linspace(0.7, 1.4, D)
            t[name + ".norm"][D - 1] = 1.0

    spec = _spec(H, G, D, E, R, window, width, scale)
    part = MIXERS.build(spec.kind, spec)
    w = _bind(part, dtype, seed=5, std=0.1, edit=edit)
    assert "sink" not in w
    h = torch.randn(T, width, generator=torch.Generator().manual_seed(9))
    h[:, 0], h[:, 1] = 1.0, 0.0
    h[marked, 1] = 1.0
    h = h.to(torch.bfloat16).float()
    cfg = _cfg(H, G, D, E, R, window, scale)
    ref = plain.attention(h.double(), w, cfg, 1e-5, "")
    steps = StepsWithValues(dtype, part.cache_need(), page, 3, T + page)
    got = _run_part(part, steps, [[(2, n)] for n in _cuts(T, how)], {2: h}, width,
                    LayerBinding(group=0, slot=0, write=True))[2]
    for j in marked:
        for i in (j, j + (window or T) - 1, j + (window or T), T - 1):
            if i < T:
                assert rel(got[i], ref[i]) < TOL[dtype], (how, "key", j, "row", i)
    assert rel(got, ref) < TOL[dtype]
    # a window that is one token off changes the row where a marked key leaves
    j = marked[-1]
    if window and 1 < window and j + window < T:
        longer = plain.attention(h.double(), w, dict(cfg, mask={"size": window + 1}), 1e-5, "")
        assert rel(longer[j + window], ref[j + window]) > 0.05


@pytest.mark.parametrize("dtype,D,E,tensor_cores", KINDS)
@pytest.mark.parametrize("how", ["prompt", "portions", "decode"])
def test_sink_gate_and_rotation(dtype, D, E, tensor_cores, how, monkeypatch):
    """Scores around and far below 0 (the added one takes most of the weight), a window over several
    pages, gates from shut to open, several requests in one step; what is left out would show."""
    from crucible_b200.ops import sink_attention as k
    from crucible_b200.parts import MIXERS, LayerBinding
    monkeypatch.setattr(k, "TENSOR_CORES", tensor_cores)
    H, G, R, width, window, scale = 6, 3, D // 4 * 2, 64, 45, 2.5 / D ** 0.5
    spec = _spec(H, G, D, E, R, window, width, scale)
    part = MIXERS.build(spec.kind, spec)

    def edit(t):
        t["g"] *= 3.0
        t["q.norm"], t["k.norm"] = torch.linspace(0.5, 1.5, D), torch.linspace(1.3, 0.6, D)
    w = _bind(part, dtype, seed=7, std=0.2, edit=edit)
    lengths = {0: 130, 1: 61, 2: 97}
    h_of = {s: torch.randn(n, width, generator=torch.Generator().manual_seed(s)).to(torch.bfloat16).float()
            for s, n in lengths.items()}
    cuts = {s: _cuts(n, how) for s, n in lengths.items()}
    schedule = []
    while any(cuts.values()):
        schedule.append([(s, cuts[s].pop(0)) for s in (1, 0, 2) if cuts[s]])
    steps = StepsWithValues(dtype, part.cache_need(), 16, 3, 144, seed=1)
    got = _run_part(part, steps, schedule, h_of, width, LayerBinding(group=0, slot=0, write=True))
    cfg = _cfg(H, G, D, E, R, window, scale)
    for s, h in h_of.items():
        assert rel(got[s], plain.attention(h.double(), w, cfg, 1e-5, "")) < TOL[dtype], s
    h = h_of[0].double()
    ref = plain.attention(h, w, cfg, 1e-5, "")
    for change in ({"g": w["g"] * 0}, {"q.norm": w["q.norm"] * 0 + 1}, {"k.norm": w["k.norm"] + 1}):
        assert rel(plain.attention(h, dict(w, **change), cfg, 1e-5, ""), ref) > 0.03, change.keys()
    for other in (dict(cfg, rot=dict(cfg["rot"], scaling=None)), dict(cfg, rot=dict(cfg["rot"], dims=R - 2))):
        assert rel(plain.attention(h, w, other, 1e-5, ""), ref) > 0.03
    monkeypatch.setattr(plain, "softmax_plus_one", lambda s, seen: torch.softmax(s.masked_fill(~seen, -1e30), -1))
    assert rel(plain.attention(h, w, cfg, 1e-5, ""), ref) > 0.03


@pytest.mark.parametrize("D", [64, 128])
def test_the_tcgen05_attention_takes_the_gate(D, monkeypatch):
    """A long prompt of two requests on the tcgen05 tiles, the gate in their epilogue: the same as the
    mma.sync tiles and as the plain function."""
    from crucible_b200.ops import tensor_core
    from crucible_b200.parts import MIXERS, LayerBinding
    H, G, width, window = 8, 2, 64, 200
    spec = _spec(H, G, D, D, D // 2, window, width, 1.5 / D ** 0.5)
    part = MIXERS.build(spec.kind, spec)
    w = _bind(part, torch.bfloat16, seed=3, std=0.2)
    h_of = {s: torch.randn(n, width).to(torch.bfloat16).float() for s, n in ((0, 600), (1, 333))}
    schedule = [[(0, 300), (1, 40)], [(0, 300), (1, 293)]]
    results, taken = [], []
    real = tensor_core._attention_tcgen05

    def watched(*args, **kw):
        ok = real(*args, **kw)
        taken.append(bool(ok) and kw.get("gate") is not None)
        return ok
    monkeypatch.setattr(tensor_core, "_attention_tcgen05", watched)
    for use in (True, False):
        monkeypatch.setattr(tensor_core, "USE_TCGEN05_ATTENTION", use)
        steps = StepsWithValues(torch.bfloat16, part.cache_need(), 16, 2, 608, seed=2)
        results.append(_run_part(part, steps, schedule, h_of, width, LayerBinding(group=0, slot=0, write=True)))
    assert taken == [True, True]
    cfg = _cfg(H, G, D, D, D // 2, window, 1.5 / D ** 0.5)
    for s, h in h_of.items():
        ref = plain.attention(h.double(), w, cfg, 1e-5, "")
        for r in results:
            assert rel(r[s], ref) < TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [3, 150])
@pytest.mark.parametrize("H,G,D,E,R,normed", [
    (4, 2, 16, 24, 8, True), (3, 1, 96, 40, 96, True), (8, 2, 128, 128, 64, True), (5, 5, 10, 6, 4, False),
    (2, 2, 320, 64, 40, True), (2, 1, 20, 512, 0, True), (3, 3, 15, 8, 6, True), (2, 1, 600, 8, 600, False)])
def test_preparation_of_neighbouring_pairs(dtype, rows, H, G, D, E, R, normed):
    """q in place, k and v in the pages, at rows few and many; sizes that the pair kernel takes and odd
    or long ones that it leaves to the general one; without a write only q is turned."""
    from crucible_b200.ops import sink_attention as k
    from crucible_b200.parts import CacheNeed, LayerBinding
    g = torch.Generator().manual_seed(2)
    width = H * D + G * (D + E) + (3 if D % 2 else 4)
    proj = torch.randn(rows, width, generator=g).to(torch.bfloat16)
    q_gain, k_gain = torch.rand(D, generator=g) + 0.5, torch.rand(D, generator=g) + 0.5
    freq = plain.turning_rates(R, 30.0).float() if R else None
    steps = StepsWithValues(dtype, CacheNeed(kv_heads=G, head_dim=D, value_dim=E), 8, 2, 200, seed=4)
    steps.fed[1] = 13
    pos = torch.arange(13, 13 + rows)
    p = proj.double()

    def heads(x, n, gain):
        x = x.reshape(rows, n, D)
        x = plain.head_norm(x, gain.double(), 1e-5) if normed else x
        return plain.turn_neighbours(x, pos, R, 30.0) if R else x
    want_q, want_k = heads(p[:, :H * D], H, q_gain), heads(p[:, H * D:(H + G) * D], G, k_gain)
    want_v = p[:, (H + G) * D:(H + G) * D + G * E].reshape(rows, G, E)
    tol = 2e-5 if dtype == torch.float32 else 8e-3          # (angles up to 160 rad, each a float32 product)
    for write in (True, False):
        binding = LayerBinding(group=0, slot=0, write=write)
        steps.fed[1] = 13
        ctx = steps.ctx([(1, rows)], binding)
        rows_in = proj.to(dtype).to(DEV).contiguous()
        keys, values = steps.storage.keys(0), steps.storage.values(0)
        keys.zero_(), values.zero_()
        k.norm_rotate_append(rows_in, q_gain.to(DEV) if normed else None, k_gain.to(DEV) if normed else None, 1e-5,
                             freq.to(DEV) if R else None, R, False, H, G, D, E, None, ctx, steps.storage, binding)
        assert rel(rows_in[:, :H * D].reshape(rows, H, D), want_q) < tol
        assert torch.equal(rows_in[:, H * D:].cpu(), proj.to(dtype)[:, H * D:])          # nothing else is touched
        if not write:
            assert not bool(keys.any()) and not bool(values.any())
            continue
        table = steps.tables[1].long()
        page, place = table[pos // 8], pos % 8
        assert rel(keys.cpu()[page, :, place], want_k) < tol
        assert torch.equal(values.cpu()[page, :, place].double(), want_v)


# ---------------------------------------------------------------------------
# experts: sigmoid scores with a correction, groups by their two best, a shared expert without a gate
# ---------------------------------------------------------------------------

def _moe_part(experts, top, ff, width, groups, shared, open_sum=True):
    from crucible_b200.config.model_config import FeedForwardSpec
    from crucible_b200.parts import FEED_FORWARDS
    return FEED_FORWARDS.build("moe", FeedForwardSpec(
        kind="moe", width=width, intermediate=ff,
        extra=(("experts", experts), ("top", top), ("groups", groups), ("shared_intermediate", shared),
               ("score", "sigmoid"), ("group_score", "two_best"), ("open_sum", open_sum))))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,ff,width,groups,shared", [
    (6, 3, 40, 48, (3, 2), 60), (8, 3, 24, 64, (4, 2), 24), (12, 4, 64, 128, (3, 1), 16), (40, 5, 16, 32, (10, 3), 130),
    (4, 1, 64, 128, (4, 1), None), (5, 2, 20, 24, None, 20), (64, 6, 8, 40, (8, 4), 8), (1, 1, 16, 32, (1, 1), 7),
    (250, 8, 8, 40, (125, 5), 264)])               # too many slices to ride along: the shared expert apart
@pytest.mark.parametrize("rows", [1, 5, 24, 90, 400])
def test_experts_by_corrected_sigmoids(dtype, experts, top, ff, width, groups, shared, rows):
    part = _moe_part(experts, top, ff, width, groups, shared)

    def edit(t):
        # corrections larger than the scores' differences, all choice scores below 0.  In bfloat16 the
        # experts lie far apart, so that the rounding of the rows decides no choice
        t["correction"] = torch.linspace(-2.0, -1.1, experts)[torch.randperm(experts, generator=torch.Generator().manual_seed(3))]
        if dtype == torch.bfloat16:
            t["router"] *= 0.001
    w = _bind(part, dtype, seed=4, std=0.3, edit=edit)
    mlp = {"router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None},
           "shared": {"ff": shared} if shared else None}
    h = torch.randn(rows, width, generator=torch.Generator().manual_seed(8)).to(torch.bfloat16).float()
    ref = plain.mixture(h.double(), w, mlp, "")
    first = None
    for as_prompt in (True, False):                     # the same rows as a portion, and as decoded tokens
        res = torch.zeros(rows, width, device=DEV)
        entries = [(0, rows)] if as_prompt else [(i, 1) for i in range(rows)]
        part.forward(Steps(dtype, n_slots=max(4, rows)).ctx(entries, None), h.to(dtype).to(DEV), res)
        assert rel(res, ref) < TOL[dtype], as_prompt
        assert part.count.tolist() == [0] * part.count.numel()          # left ready for the next step
        if dtype == torch.float32 and first is not None:
            assert torch.equal(res, first)
        first = res
    if top < experts and rows > 1:
        assert rel(plain.mixture(h.double(), dict(w, correction=w["correction"] * 0), mlp, ""), ref) > 1e-2


def test_a_shared_expert_beside_the_sum_is_the_same():
    """The shared expert as a feed-forward of its own behind the experts, without an open sum."""
    h = torch.randn(70, 64, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).float()
    out = []
    for open_sum in (True, False):
        part = _moe_part(8, 2, 32, 64, (4, 2), 48, open_sum)
        w = _bind(part, torch.float32, seed=2, std=0.3)
        res = torch.zeros(70, 64, device=DEV)
        part.forward(Steps(torch.float32).ctx([(0, 70)], None), h.to(DEV), res)
        mlp = {"router": {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 2}}, "shared": {"ff": 48}}
        assert rel(res, plain.mixture(h.double(), w, mlp, "")) < TOL[torch.float32]
        out.append(res)


def _route(logits, top, n, ns=0, **kw):
    from crucible_b200.ops import moe as k
    t = logits.shape[0]
    tiles = k.max_tiles(t, top + ns, n + ns)
    pairs = t * (top + ns)
    idx, place, order = (torch.zeros(pairs, dtype=torch.int32, device=DEV) for _ in range(3))
    weight = torch.zeros(pairs, device=DEV)
    count = torch.zeros(n + ns, dtype=torch.int32, device=DEV)
    plan = torch.zeros(k.plan_ints(n + ns, tiles), dtype=torch.int32, device=DEV)
    k.route(logits, top, idx, weight, place, count, plan, tiles, order, n_experts=n, n_shared=ns, **kw)
    assert count.tolist() == [0] * (n + ns) and sorted(order.tolist()) == list(range(pairs))
    return idx.view(t, -1).tolist(), weight.view(t, -1).cpu()


def test_the_choice_in_the_routing_kernel():
    """The best single expert's group loses to the group with the best two; negative scores; the lower
    group and expert on ties; weights without the correction; a shared expert's slices at weight 1."""
    from crucible_b200.ops import KernelError
    logits = torch.tensor([[3.0, -9.0, 0.5, 0.4, 0.0, -0.1],
                           [1.0, 1.0, 1.0, 1.0, 1.0, 1.0],
                           [-1.0, -2.0, -0.5, -3.0, 0.2, 0.1]], device=DEV)
    idx, weight = _route(logits, 2, 6, sigmoid=True, groups=(3, 1), group_best_two=True)
    assert idx == [[2, 3], [0, 1], [4, 5]]
    assert torch.allclose(weight, torch.sigmoid(logits.cpu().gather(1, torch.tensor(idx))))
    assert _route(logits, 2, 6, sigmoid=True, groups=(3, 1))[0][0] == [0, 1]           # by the best alone
    for shift in (-5.0, 4.0):           # a correction common to all changes nothing, whatever its sign
        c = torch.full((6,), shift, device=DEV)
        assert _route(logits, 2, 6, sigmoid=True, correction=c, groups=(3, 1), group_best_two=True)[0] == idx
    c = torch.tensor([0.0, 0.0, 0.0, 0.0, -1.0, 0.5], device=DEV)
    i2, w2 = _route(logits, 3, 6, 2, sigmoid=True, correction=c, groups=(3, 2), group_best_two=True)
    choice = torch.sigmoid(logits.cpu()) + c.cpu()
    assert i2 == [plain.choose_experts(row, 3, 3, 2) + [6, 7] for row in choice]
    for row, chosen in enumerate(i2):
        assert torch.allclose(w2[row, :3], torch.sigmoid(logits[row].cpu()[chosen[:3]])) and w2[row, 3:].tolist() == [1.0, 1.0]
    # groups of one expert each
    assert _route(logits, 1, 6, sigmoid=True, groups=(6, 2), group_best_two=True)[0] == [[0], [0], [4]]
    g = torch.Generator().manual_seed(5)
    for n, top, groups in ((256, 8, (8, 3)), (96, 32, (3, 2)), (33, 4, (11, 4)), (30, 7, (1, 1))):
        z, c = 2 * torch.randn(70, n, generator=g), torch.randn(n, generator=g)
        got, w = _route(z.to(DEV), top, n, sigmoid=True, correction=c.to(DEV), groups=groups, group_best_two=True)
        want = [plain.choose_experts(row, top, *groups) for row in torch.sigmoid(z.double()) + c.double()]
        assert got == want
        assert torch.allclose(w, torch.sigmoid(z.gather(1, torch.tensor(want))), atol=1e-6)
    with pytest.raises(KernelError):
        _route(logits, 2, 6, correction=torch.zeros(6, device=DEV))


# ---------------------------------------------------------------------------
# the end of a layer, the entry of a pass
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("width", [40, 43, 1000, 1028, 2048, 4100, 9000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_close(width, dtype):
    from crucible_b200.ops import layer_close as k
    t, top, g = 5, 3, torch.Generator().manual_seed(width)

    def rnd(*shape):
        return torch.randn(*shape, generator=g).to(DEV)
    x, mixer, shared = rnd(t, width), rnd(t, width), rnd(t, width)
    rows, gate, s1, s2, g1, g2 = rnd(t * top, width), rnd(t), rnd(width), rnd(width), rnd(width), rnd(width)
    d = lambda v: v.double().cpu()
    tol = 3e-6 if dtype == torch.float32 else 6e-3
    # the rows of the sorted order: place of pair p is offsets[idx] + place
    order = torch.randperm(t * top, generator=g)
    plan = _i32([1, 0, t * top])
    by_plan = (plan, torch.zeros(t * top, dtype=torch.int32, device=DEV), order.to(torch.int32).to(DEV), rnd(t * top))
    pairs = d(rows).view(t, top, width).sum(1)
    sorted_sum = (d(rows)[order] * d(by_plan[3])[:, None]).view(t, top, width).sum(1)
    cases = [
        (mixer, s1, k.OpenSum(rows, top, None, shared, gate), s2, d(s1) * d(mixer) + d(s2) * (pairs + d(gate)[:, None] * d(shared))),
        (mixer, s1, k.OpenSum(rows, top, by_plan, shared, None), s2, d(s1) * d(mixer) + d(s2) * (sorted_sum + d(shared))),
        (mixer, None, k.OpenSum(rows, top, None, None, None), None, d(mixer) + pairs),
        (None, None, k.OpenSum(None, 0, None, shared, None), s2, d(s2) * d(shared)),
        (mixer, s1, None, None, d(s1) * d(mixer)),
        (None, None, None, None, torch.zeros(t, width, dtype=torch.float64))]
    for i, (m, a, o, b, add) in enumerate(cases):
        want = d(x) + add
        for gains in ((), (g1,), (g1, g2)):
            y = x.clone()
            outs = [torch.empty(t, width, dtype=dtype, device=DEV) for _ in gains]
            eps = (1e-5, 0.3)
            k.close(y, m, a, o, b, [(gain, e, out) for gain, e, out in zip(gains, eps, outs)])
            assert rel(y, want) < 3e-6, i
            for gain, e, out in zip(gains, eps, outs):
                assert rel(out, plain.unit_rms(want, e) * d(gain)) < tol, i
            # taken in the same launch or in one of their own, the norms are the same bits
            alone = [torch.empty_like(out) for out in outs]
            if alone:
                k.close(y, None, None, None, None, [(gain, e, out) for gain, e, out in zip(gains, eps, alone)])
                assert all(torch.equal(p, q) for p, q in zip(outs, alone)), i


def test_layer_close_refuses():
    from crucible_b200.ops import KernelError, layer_close as k
    x = torch.zeros(4, 16, device=DEV)
    v = torch.zeros(16, device=DEV)
    out = torch.zeros(4, 16, device=DEV)
    with pytest.raises(KernelError):
        k.close(x, x.bfloat16(), None, None, None)
    with pytest.raises(KernelError):
        k.close(x, None, v[:8], None, None)
    with pytest.raises(KernelError):
        k.close(x, None, None, k.OpenSum(torch.zeros(7, 16, device=DEV), 2), None)
    with pytest.raises(KernelError):
        k.close(x, None, None, None, None, [(v, 1e-5, out)] * 3)
    with pytest.raises(KernelError):
        k.swap_rows(x, out[:2].contiguous())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,rows", [(44, 3), (64, 1), (128, 150), (96, 40)])
def test_entry_of_a_pass(dtype, width, rows):
    from crucible_b200.models.decoder import ModelMatrices
    part = ModelMatrices(("in",), width)
    g = torch.Generator().manual_seed(3)
    w = (0.2 * torch.randn(width, 2 * width, generator=g)).to(torch.bfloat16)
    part.bind({"in": w.to(dtype).to(DEV)}, dtype, torch.device(DEV))
    x0 = torch.randn(rows, width, generator=g)
    ctx = Steps(dtype).ctx([(0, rows)], None)
    x = x0.to(DEV)
    share = part.of_embedding(ctx, "in", x)
    assert torch.equal(x.cpu(), x0)
    want = x0.double()
    for _ in range(3):                              # three passes, the embedding's share taken once
        part.enter(ctx, "in", x, share)
        want = plain.enter_pass(want, x0.double(), w.double())
        assert x.dtype == torch.float32
        assert rel(x, want) < (1e-5 if dtype == torch.float32 else 2e-2)
        x.add_(1.0)
        want = want + 1.0
    assert rel(plain.enter_pass(x0.double(), x0.double() * 0, w.double()), plain.enter_pass(x0.double(), x0.double(), w.double())) > 0.1


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_scaled_embedding_is_the_head_without_its_scale(dtype, tmp_path):
    """The head's logits come from the table as it is stored."""
    import gavipel_cases as cases
    from crucible_b200.config import parse_config
    from crucible_b200.models.decoder import DecoderModel
    config = cases.model(50, 32, 1e-5, 13.0, [cases.attention(1, 1, 8, 8, 0.3, 4, None, None)], None)
    model = DecoderModel(parse_config(config))
    table = (torch.randn(50, 32, generator=torch.Generator().manual_seed(1)) * 0.3).to(torch.bfloat16)
    model.embedding.bind({"table": table.to(dtype).to(DEV)}, dtype, torch.device(DEV))
    model.head.tie(model.embedding.table)
    ctx = Steps(dtype).ctx([(0, 4)], None)
    ids = [3, 49, 0, 3]
    x = model.embedding.forward(ctx, _i32(ids))
    assert rel(x, table.double()[ids] * 13.0) < 1e-6
    rows = torch.randn(4, 32, generator=torch.Generator().manual_seed(2)).to(torch.bfloat16)
    logits = model.head.forward(ctx, rows.to(dtype).to(DEV))
    assert rel(logits, rows.double() @ table.double().T) < 1e-5
