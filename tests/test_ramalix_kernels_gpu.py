"""Each mechanism of the Ramalix design alone: its part, driven over hand-made steps, against the
one-mechanism functions of `plain_ramalix.py`.  Inputs are made so that a fault shows: marked keys
whose scores stand out at every chunk's and page's edge, sinks that take most of a head's weight,
sharp softmaxes that find one key far back, decays at both ends, routers that prefer experts of
groups that are not kept."""
import pytest
import torch

import plain_ramalix as plain
from test_futepel_kernels_gpu import DEV, TOL, Steps, _bind, _binding, _check_mixer, _cut, rel
from test_nipapel_kernels_gpu import StepsWithValues, _cuts, _run_part

pytestmark = pytest.mark.gpu


# ---------------------------------------------------------------------------
# the norm with one number, the input convolution, the embedding taken again, the logits' scale
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_with_one_number(dtype):
    from crucible_b200.config.model_config import NormSpec
    from crucible_b200.parts import NORMS
    norm = NORMS.build("rmsnorm_one_number", NormSpec(kind="rmsnorm_one_number", width=72, eps=1e-5))
    assert [tuple(d.shape) for d in norm.tensors()] == [()]
    norm.bind({"gain": torch.tensor(1.75, device=DEV)}, dtype, torch.device(DEV))
    x = torch.randn(9, 72) * 3.0
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    assert rel(norm.forward(Steps(dtype).ctx([(0, 9)], None), x.to(DEV)), plain.norm_one_number(x.double(), 1.75, 1e-5)) < tol
    norm.scale_gain(0.5)
    assert rel(norm.forward(Steps(dtype).ctx([(0, 9)], None), x.to(DEV)), plain.norm_one_number(x.double(), 0.875, 1e-5)) < tol


def _run_norm_conv(x_of, gain, eps, w, dtype, schedule, steps, width):
    """`x_of`: slot -> rows; returns every slot's results over the schedule."""
    from crucible_b200.ops import input_conv
    out = {}
    for entries in schedule:
        ctx = steps.ctx(entries, None)
        x = torch.cat([x_of[slot][steps.fed[slot] - n:steps.fed[slot]] for slot, n in entries], 0).to(DEV).contiguous()
        y = torch.full(x.shape, 7.0, device=DEV, dtype=dtype)
        input_conv.norm_conv(x, gain, eps, w, ctx, steps.state, 16, y)
        at = 0
        for slot, n in entries:
            out.setdefault(slot, []).append(y[at:at + n].clone())
            at += n
    torch.cuda.synchronize()
    return {slot: torch.cat(chunks, 0) for slot, chunks in out.items()}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,taps", [(40, 4), (45, 3), (256, 2), (1100, 4), (64, 1), (36, 5), (50, 12), (2304, 3)])
def test_norm_and_input_convolution(dtype, width, taps):
    g = torch.Generator().manual_seed(3)
    w = torch.randn(width, taps, generator=g)
    gain, eps = 1.3, 1e-5
    lengths = {0: 70, 1: 5, 3: 23}
    x_of = {slot: torch.randn(n, width, generator=g) * 2.0 for slot, n in lengths.items()}
    ref = {slot: plain.input_conv(plain.norm_one_number(x.double(), gain, eps), w.double()) for slot, x in x_of.items()}
    wd, gd = w.t().contiguous().to(DEV), torch.full((width,), gain, device=DEV)
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    steps = Steps(dtype, state_bytes=16 + 4 * max(1, taps - 1) * width)
    whole = None
    mixed = {slot: _cut(n, [2, 1, 9, 3, 17]) for slot, n in lengths.items()}
    schedules = {"whole": [[(slot, n)] for slot, n in lengths.items()],
                 "single": [[(0, 1), (1, 1), (3, 1)]] * 5 + [[(3, 1), (0, 1)]] * 18 + [[(0, 1)]] * 47,
                 "mixed": []}
    while any(mixed.values()):
        schedules["mixed"].append([(slot, c.pop(0)) for slot, c in sorted(mixed.items(), reverse=True) if c])
    for label, schedule in schedules.items():
        got = _run_norm_conv(x_of, gd, eps, wd, dtype, schedule, steps, width)
        for slot in lengths:
            assert rel(got[slot], ref[slot]) < tol, (label, slot)
            if whole is not None:
                assert torch.equal(got[slot], whole[slot]), (label, slot)      # the same bits however it is cut
            steps.free(slot)                       # the next schedule finds the slot as it is handed out
        whole = whole or got
    # a convolution that is one token off, or that forgets the rows before a portion, shows
    if taps > 1:
        h = plain.norm_one_number(x_of[0].double(), gain, eps)
        assert rel(plain.input_conv(h, w.double().roll(1, 1)), ref[0]) > 0.1


def test_a_slot_that_is_not_clean_would_show():
    """The convolution's inputs are state: with another request's rows left in the slot the first
    tokens differ."""
    width, taps = 40, 4
    x = torch.randn(6, width)
    w = torch.randn(taps, width, device=DEV)
    steps = Steps(torch.float32, state_bytes=16 + 4 * (taps - 1) * width)
    gain = torch.ones(width, device=DEV)
    first = _run_norm_conv({0: x}, gain, 1e-5, w, torch.float32, [[(0, 6)]], steps, width)[0]
    steps.fed[0] = 0                                # taken again without being cleaned
    again = _run_norm_conv({0: x}, gain, 1e-5, w, torch.float32, [[(0, 6)]], steps, width)[0]
    assert not torch.equal(first[:taps - 1], again[:taps - 1]) and torch.equal(first[taps - 1:], again[taps - 1:])


def test_rows_and_a_vector_added_to_the_residual():
    from crucible_b200 import ops
    x, rows, v = torch.randn(33, 52), torch.randn(33, 52), torch.randn(52)
    got = x.to(DEV)
    ops.add_rows(got, rows.to(DEV), v.to(DEV))
    assert torch.equal(got.cpu(), (x + rows) + v)
    got = x.to(DEV)
    ops.add_rows(got, rows.to(DEV))
    assert torch.equal(got.cpu(), x + rows)
    with pytest.raises(ops.KernelError):
        ops.add_rows(got, rows[:5].to(DEV))


# ---------------------------------------------------------------------------
# differential attention
# ---------------------------------------------------------------------------

def _diff_spec(H, G, D, E, width, scale, diff, temp, out_scale=1.0):
    from crucible_b200.config.model_config import MixerSpec
    return MixerSpec(kind="differential_attention", width=width, n_heads=H, n_kv_heads=G, head_dim=D,
                     softmax_scale=scale, extra=(("value_dim", E), ("diff", diff), ("norm_eps", 1e-5),
                                                 ("q_temp", temp), ("out_scale", out_scale)))


def _diff_cfg(H, G, D, E, scale, diff, temp):
    return {"heads": H, "kv_heads": G, "dim": D, "vdim": E, "scale": scale, "diff": diff,
            "q_temp": {"coef": temp[0], "every": temp[1]} if temp else None}


def _beside(cuts, slot, length, each):
    """Steps of slot 0's portions `cuts`, with up to `each` tokens of another request in front of
    every one of them until its `length` tokens are through."""
    schedule, left = [], length
    for n in cuts:
        entry = []
        if left:
            entry.append((slot, min(left, each)))
            left -= min(left, each)
        schedule.append(entry + [(0, n)])
    while left:
        schedule.append([(slot, min(left, each))])
        left -= min(left, each)
    return schedule


@pytest.mark.parametrize("dtype,H,G,D,E,page", [
    (torch.float32, 4, 2, 16, 24, 8), (torch.float32, 3, 1, 10, 20, 16),
    (torch.bfloat16, 3, 1, 10, 14, 16),              # CUDA cores: no multiples of 16
    (torch.bfloat16, 4, 2, 8, 16, 8),                # keys of both maps as wide as a value: paged attention
    (torch.bfloat16, 4, 2, 32, 64, 16), (torch.bfloat16, 2, 2, 64, 128, 16),       # ... on the tcgen05 tiles
    (torch.bfloat16, 4, 1, 24, 16, 16), (torch.bfloat16, 2, 1, 16, 112, 32)])      # ... of unlike sizes
@pytest.mark.parametrize("how", ["prompt", "portions", "decode"])
def test_differential_attention(dtype, H, G, D, E, page, how):
    from crucible_b200.parts import MIXERS
    width, T, diff, temp = 48, 330, 0.6, (0.3, 40)
    scale = 2.0 / (0.3 * 0.3 * width * D ** 0.5)             # scores of spread 2
    part = MIXERS.build("differential_attention", _diff_spec(H, G, D, E, width, scale, diff, temp, 0.7))

    def edit(t):
        # a lambda far from the layer's constant, biases as large as the projections
        t["lq1"], t["lk1"] = torch.full((D,), 0.5), torch.full((D,), 1.0 / D)
        t["lq2"], t["lk2"] = torch.full((D,), -0.5), torch.full((D,), 2.0 / D)
        for name in ("q.b", "k.b", "v.b"):
            t[name] = t[name] * 10
    w = _bind(part, dtype, 5, std=0.3, edit=edit)
    steps = StepsWithValues(dtype, part.cache_need(), page, 2, 512, seed=3)
    h_of = {0: torch.randn(T, width).to(torch.bfloat16).float(), 1: torch.randn(90, width).to(torch.bfloat16).float()}
    got = _run_part(part, steps, _beside(_cuts(T, how), 1, 90, 1 if how != "decode" else 7), h_of, width,
                    _binding(part, group=0))
    cfg = _diff_cfg(H, G, D, E, scale, diff, temp)
    for slot, h in h_of.items():
        ref = 0.7 * plain.differential_attention(h.double(), w, cfg, 1e-5, "")
        # (the difference of two nearly equal means is normed: bfloat16's rounding of the means is)
        assert rel(got[slot], ref) < (TOL[dtype] if dtype == torch.float32 else 5e-2), (slot, how)
    # each of its parts is seen (all but the keys' bias, which adds one number to all of a row's scores)
    h = h_of[0].double()
    ref = plain.differential_attention(h, w, cfg, 1e-5, "")
    for change in ({"lq1": w["lq1"] * 0}, {"q.b": w["q.b"] * 0}, {"v.b": w["v.b"] * 0},
                   {"o.b": w["o.b"] * 0}):
        assert rel(plain.differential_attention(h, dict(w, **change), cfg, 1e-5, ""), ref) > 1e-2, change.keys()
    assert rel(plain.differential_attention(h, w, dict(cfg, q_temp=None), 1e-5, ""), ref) > 0.05


@pytest.mark.parametrize("dtype,H,G,D,E", [(torch.float32, 2, 1, 12, 20), (torch.bfloat16, 4, 2, 32, 64),
                                           (torch.bfloat16, 2, 2, 16, 48), (torch.bfloat16, 2, 1, 64, 128)])
@pytest.mark.parametrize("how", ["prompt", "portions", "decode"])
def test_each_map_finds_keys_of_its_own_far_back(dtype, H, G, D, E, how):
    """Map 1 is held by one set of marked tokens, map 2 by another: their keys stand out in that
    map alone, at page borders and far back; swapping the maps or losing a key shows."""
    from crucible_b200.parts import MIXERS
    width, T, page = 48, 300, 8
    part = MIXERS.build("differential_attention", _diff_spec(H, G, D, E, width, 1.0, 0.4, None))
    one, two = [3, 7, 64, 201], [8, 100, 255]

    def edit(t):
        for name in ("q", "k", "v"):
            t[name][:, 0:3] = 0.0
            t[name + ".b"] *= 0.1
        t["q"].view(H, 2, D, width)[:, :, 0, :] = 0.0
        t["q"].view(H, 2, D, width)[:, :, 0, 0] = 3.0            # every query asks in channel 0
        t["k"].view(G, 2, D, width)[:, :, 0, :] = 0.0
        t["k"].view(G, 2, D, width)[:, 0, 0, 1] = 4.0            # map 1 answers to feature 1
        t["k"].view(G, 2, D, width)[:, 1, 0, 2] = 4.0            # map 2 to feature 2
    w = _bind(part, dtype, 2, std=0.05, edit=edit)
    h = torch.randn(T, width, generator=torch.Generator().manual_seed(9))
    h[:, 0], h[:, 1], h[:, 2] = 1.0, 0.0, 0.0
    h[one, 1] = 1.0
    h[two, 2] = 1.0
    h = h.to(torch.bfloat16).float()
    steps = StepsWithValues(dtype, part.cache_need(), page, 2, 320, seed=3)
    got = _run_part(part, steps, [[(1, n)] for n in _cuts(T, how)], {1: h}, width, _binding(part, group=0))[1]
    ref = plain.differential_attention(h.double(), w, _diff_cfg(H, G, D, E, 1.0, 0.4, None), 1e-5, "")
    tol = TOL[dtype] if dtype == torch.float32 else 5e-2
    for j in one + two:
        for i in (j, j + 1, T - 1):
            assert rel(got[i], ref[i]) < tol, (how, "key", j, "row", i)
    assert rel(got, ref) < tol
    swapped = dict(w)
    swapped["k"] = w["k"].view(G, 2, D, width).flip(1).reshape(G * 2 * D, width)
    assert rel(plain.differential_attention(h.double(), swapped, _diff_cfg(H, G, D, E, 1.0, 0.4, None), 1e-5, ""), ref) > 0.2


# ---------------------------------------------------------------------------
# chunked attention with a sink
# ---------------------------------------------------------------------------

def _chunked_spec(H, G, D, E, R, size, width, scale, out_scale=1.0):
    from crucible_b200.config.model_config import MixerSpec, PositionSpec
    position = PositionSpec(kind="rope_interleaved", rotary_dim=R, theta=700.0, max_positions=0) if R else None
    return MixerSpec(kind="sink_attention", width=width, n_heads=H, n_kv_heads=G, head_dim=D, softmax_scale=scale,
                     window=size, position=position,
                     extra=(("value_dim", E), ("keep_first", 0), ("sink", True), ("gate", None),
                            ("value_norm_eps", None), ("qk_norm_eps", None), ("chunked", True),
                            ("out_scale", out_scale)))


@pytest.mark.parametrize("dtype,D,E,tensor_cores", [
    (torch.float32, 16, 24, False), (torch.bfloat16, 20, 12, False), (torch.bfloat16, 32, 32, False),
    (torch.bfloat16, 32, 32, True), (torch.bfloat16, 48, 16, True), (torch.bfloat16, 16, 80, True),
    # heads of 64 and 128: portions of 32 tokens and more on the tcgen05 tiles
    (torch.bfloat16, 64, 64, True), (torch.bfloat16, 128, 128, True)])
@pytest.mark.parametrize("how", ["prompt", "portions", "decode"])
@pytest.mark.parametrize("size,T", [(10, 90), (70, 300), (128, 300), (1, 20), (500, 120)])
def test_chunked_attention_sees_exactly_its_keys(dtype, D, E, tensor_cores, how, size, T, monkeypatch):
    """Feature 0 of the input is 1 for every token and feature 1 for a few marked tokens; a channel
    that is not turned makes a marked key's score stand out.  They are the first and the last tokens
    of chunks and the tokens at page borders: every row of the chunk is held by them, no row of the
    next chunk is.  The sink takes nearly all of the first head's weight and none of the last's."""
    from crucible_b200.ops import sink_attention as k
    from crucible_b200.parts import MIXERS, LayerBinding
    monkeypatch.setattr(k, "TENSOR_CORES", tensor_cores)
    H, G, R, width, page, scale = 4, 2, 8, 48, 8, 0.5
    marked = sorted(j for j in {0, size - 1, size, 2 * size - 1, 2 * size + 1, 3 * size + 5, 7, 8} if j < T)

    def edit(t):
        for name, heads, feature in (("q", H, 0), ("k", G, 1)):
            m = t[name].view(heads, D, width)
            m[:, :, feature] = 0.0
            m[:, D - 1, :] = 0.0
            m[:, D - 1, feature] = 4.0                        # a marked key's score: 4 * 4 * scale = 8
        t["sink"] = torch.tensor([9.0, 3.0, 0.0, -6.0])
    spec = _chunked_spec(H, G, D, E, R, size, width, scale, 1.5)
    part = MIXERS.build(spec.kind, spec)
    w = _bind(part, dtype, seed=5, std=0.1, edit=edit)
    h = torch.randn(T, width, generator=torch.Generator().manual_seed(9))
    h[:, 0], h[:, 1] = 1.0, 0.0
    h[marked, 1] = 1.0
    h = h.to(torch.bfloat16).float()
    cfg = {"heads": H, "kv_heads": G, "dim": D, "vdim": E, "scale": scale, "rot": {"base": 700.0, "dims": R},
           "mask": {"size": size}}
    ref = 1.5 * plain.chunked_attention(h.double(), w, cfg, 1e-5, "")
    assert part.cache_need().window == size and part.cache_need().chunked
    steps = StepsWithValues(dtype, part.cache_need(), page, 3, T + page)
    got = _run_part(part, steps, [[(2, n)] for n in _cuts(T, how)], {2: h}, width,
                    LayerBinding(group=0, slot=0, write=True))[2]
    for j in marked:
        last = j // size * size + size - 1                      # the last row that sees key j
        for i in (j, last, last + 1, T - 1):
            if i < T:
                assert rel(got[i], ref[i]) < TOL[dtype], (how, "key", j, "row", i)
    assert rel(got, ref) < TOL[dtype]
    if 1 < size < T:
        # chunks that begin one token late, and a softmax without the sink, give other results
        late = 1.5 * plain.chunked_attention(h.double(), w, dict(cfg, mask={"size": size + 1}), 1e-5, "")
        assert rel(late, ref) > 0.05
        gone = dict(w)
        gone["sink"] = torch.full((H,), -60.0).double()
        assert rel(1.5 * plain.chunked_attention(h.double(), gone, cfg, 1e-5, ""), ref) > 0.05


@pytest.mark.parametrize("D", [64, 128])
def test_unequal_portions_in_one_step_of_chunked_attention(D):
    """Portions of three requests, all on the tcgen05 tiles, that begin in the middle of chunks."""
    from crucible_b200.parts import MIXERS, LayerBinding
    H, G, size, width, page = 4, 2, 90, 64, 16
    spec = _chunked_spec(H, G, D, D, 32, size, width, 0.4)
    part = MIXERS.build(spec.kind, spec)
    w = _bind(part, torch.bfloat16, seed=7, std=0.15)
    lengths = {0: 400, 1: 150, 2: 333}
    h_of = {s: torch.randn(n, width).to(torch.bfloat16).float() for s, n in lengths.items()}
    cuts = {0: [100, 170, 130], 1: [40, 60, 50], 2: [89, 2, 242]}
    schedule = [[(s, cuts[s][i]) for s in (1, 0, 2)] for i in range(3)]
    steps = StepsWithValues(torch.bfloat16, part.cache_need(), page, 3, 416, seed=1)
    got = _run_part(part, steps, schedule, h_of, width, LayerBinding(group=0, slot=0, write=True))
    cfg = {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": 0.4, "rot": {"base": 700.0, "dims": 32},
           "mask": {"size": size}}
    for s, h in h_of.items():
        assert rel(got[s], plain.chunked_attention(h.double(), w, cfg, 1e-5, "")) < TOL[torch.bfloat16], s


# ---------------------------------------------------------------------------
# the delta rule with a decay per key channel
# ---------------------------------------------------------------------------

def _delta_spec(H, G, D, E, taps, width, rank, out_scale=1.0):
    from crucible_b200.config.model_config import MixerSpec
    return MixerSpec(kind="channel_delta", width=width, n_heads=H, n_kv_heads=G, head_dim=D,
                     extra=(("value_dim", E), ("conv_taps", taps), ("norm_eps", 1e-5), ("rank", rank),
                            ("out_scale", out_scale)))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,taps,width,rank", [
    (4, 2, 16, 24, 4, 40, 5), (3, 3, 10, 6, 3, 44, 8), (2, 1, 64, 64, 2, 128, 16),
    (6, 2, 36, 20, 1, 64, 3), (2, 2, 128, 48, 4, 64, 24), (1, 1, 200, 16, 5, 32, 7), (8, 1, 32, 128, 11, 48, 1)])
def test_channel_delta(dtype, H, G, D, E, taps, width, rank):
    spec = _delta_spec(H, G, D, E, taps, width, rank, 0.6)
    cfg = {"heads": H, "kv_heads": G, "dim": D, "vdim": E}

    def edit(t):
        # decays from nearly 1 (channels that remember everything) to nearly 0, some strongly driven
        # by the input
        t["dt_bias"] = torch.linspace(-7.0, 3.0, H * D)[torch.randperm(H * D, generator=torch.Generator().manual_seed(1))]
        t["a2"] *= 3.0
    _check_mixer(spec, lambda h, w: 0.6 * plain.channel_delta(h, w, cfg, 1e-5, ""), dtype, {0: 83, 2: 7, 3: 1},
                 edit=edit)


def test_channel_delta_state_is_used_again_clean():
    from crucible_b200.parts import MIXERS
    spec = _delta_spec(2, 1, 24, 16, 3, 40, 4)
    cfg = {"heads": 2, "kv_heads": 1, "dim": 24, "vdim": 16}
    part = MIXERS.build(spec.kind, spec)
    w = _bind(part, torch.float32, 4)
    steps = Steps(torch.float32, state_bytes=part.state_bytes(), n_slots=2)
    a, b = (torch.randn(n, 40).to(torch.bfloat16).float() for n in (50, 31))
    _run_part(part, steps, [[(0, 50)]], {0: a}, 40, _binding(part))
    steps.free(0)
    got = _run_part(part, steps, [[(0, 20)], [(0, 2)], [(0, 9)]], {0: b}, 40, _binding(part))[0]
    assert rel(got, plain.channel_delta(b.double(), w, cfg, 1e-5, "")) < TOL[torch.float32]


@pytest.mark.parametrize("D,E,H,G", [(256, 40, 2, 2), (64, 24, 6, 3), (30, 17, 3, 1)])
def test_the_recurrence_alone_with_vector_decays(D, E, H, G):
    """The kernel by itself over prepared rows, in one piece and cut in three, decays at both ends;
    query/key heads shared by several value heads, whose decays are their own."""
    from crucible_b200.ops import recurrent as k
    from crucible_b200.parts import LayerBinding
    T = 53
    g = torch.Generator().manual_seed(5)
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)
    q, kk = (unit(torch.randn(T, G, D, generator=g)) for _ in range(2))
    v = torch.randn(T, H, E, generator=g)
    decay = torch.rand(T, H, D, generator=g) ** 0.05
    decay[:, :, 0], decay[:, :, 1] = 1.0, 0.0
    beta = torch.rand(T, H, generator=g)
    qkv = torch.cat([q.view(T, -1), kk.view(T, -1), v.view(T, -1), decay.view(T, -1)], 1).contiguous().to(DEV)
    S = torch.zeros(H, D, E, dtype=torch.float64)
    want = torch.zeros(T, H, E, dtype=torch.float64)
    qe, ke = (x.double().repeat_interleave(H // G, 1) for x in (q, kk))
    for t in range(T):
        S = decay[t].double()[:, :, None] * S
        u = beta[t].double()[:, None] * (v[t].double() - torch.einsum("hde,hd->he", S, ke[t]))
        S = S + ke[t][:, :, None] * u[:, None, :]
        want[t] = torch.einsum("hde,hd->he", S, qe[t])
    C = 2 * G * D + H * E
    results = []
    for cuts in ([T], [20, 2, 31]):
        steps = Steps(torch.float32, state_bytes=4 * H * D * E + 64)
        binding = LayerBinding(state_offset=0, state_bytes=4 * H * D * E)
        at, out = 0, []
        for n in cuts:
            ctx = steps.ctx([(1, n)], None)
            o = torch.empty(n, H * E, device=DEV)
            k.matrix_memory(k.CHANNEL, qkv[at:at + n].contiguous(), 0, G * D, 2 * G * D, None,
                            beta[at:at + n].contiguous().to(DEV), ctx, ctx.state(binding), 0, 0, 0, o, H, G, D, E, w_off=C)
            out.append(o)
            at += n
        results.append(torch.cat(out, 0))
        assert rel(results[-1].view(T, H, E), want) < 1e-5
        left = steps.state[1, :4 * H * D * E].contiguous().view(torch.float32).view(H, D, E)
        assert rel(left, S) < 1e-5
    assert torch.equal(results[0], results[1])


# ---------------------------------------------------------------------------
# experts in groups, with a gated shared expert
# ---------------------------------------------------------------------------

def _moe_part(experts, top, ff, width, groups, shared, out_scale):
    from crucible_b200.config.model_config import FeedForwardSpec
    from crucible_b200.parts import FEED_FORWARDS
    return FEED_FORWARDS.build("moe", FeedForwardSpec(
        kind="moe", width=width, intermediate=ff,
        extra=(("experts", experts), ("top", top), ("groups", groups), ("shared_intermediate", shared),
               ("shared_gate", shared is not None), ("out_scale", out_scale))))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,ff,width,groups,shared", [
    (6, 3, 40, 48, (3, 2), 60), (8, 3, 24, 64, (4, 2), 24), (12, 4, 64, 128, (3, 1), 16), (40, 5, 16, 32, (10, 3), 130),
    (4, 1, 64, 128, (4, 1), None), (5, 2, 20, 24, None, 20), (64, 6, 8, 40, (8, 4), 8), (1, 1, 16, 32, (1, 1), 7),
    (250, 8, 8, 40, (125, 5), 264)])               # too many slices to ride along: the shared expert apart
@pytest.mark.parametrize("rows", [1, 5, 90, 400])
def test_experts_in_groups_with_a_gated_shared_expert(dtype, experts, top, ff, width, groups, shared, rows):
    part = _moe_part(experts, top, ff, width, groups, shared, 0.3)
    w = _bind(part, dtype, seed=4, std=0.3)
    mlp = {"router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None},
           "shared": {"ff": shared} if shared else None}
    h = torch.randn(rows, width, generator=torch.Generator().manual_seed(8)).to(torch.bfloat16).float()
    ref = 0.3 * plain.mixture(h.double(), w, mlp, "")
    for as_prompt in (True, False):                     # the same rows as a portion, and as decoded tokens
        res = torch.zeros(rows, width, device=DEV)
        entries = [(0, rows)] if as_prompt else [(i, 1) for i in range(rows)]
        part.forward(Steps(dtype, n_slots=max(4, rows)).ctx(entries, None), h.to(dtype).to(DEV), res)
        assert rel(res, ref) < TOL[dtype], as_prompt
        assert part.count.tolist() == [0] * part.count.numel()          # left ready for the next step
        if dtype == torch.float32 and not as_prompt:
            assert torch.equal(res, first)
        first = res
    # leaving the groups or the gate out is seen
    if groups and groups[1] < min(groups[0], top) and rows > 1:      # (the best experts fill at most `top` groups)
        free = dict(mlp, router=dict(mlp["router"], groups=None))
        assert rel(0.3 * plain.mixture(h.double(), w, free, ""), ref) > 0.02
    if shared:
        open_gate = dict(w)
        open_gate["shared.sg"] = torch.zeros_like(w["shared.sg"])
        assert rel(0.3 * plain.mixture(h.double(), open_gate, mlp, ""), ref) > 1e-3


def test_groups_of_experts_in_the_routing_kernel():
    """The choice alone: the kept groups are those with the best single expert, the lower group and
    the lower expert win on equal logits, and a shared expert's slices follow with their gate."""
    from crucible_b200.ops import moe as k
    logits = torch.tensor([[5.0, -9.0, 4.0, 4.0, 4.5, 4.4, 0.0],      # groups (0,1) (2,3) (4,5): keep 0 and 2
                           [1.0, 1.0, 1.0, 1.0, 1.0, 1.0, 2.0],      # all equal: the first two groups
                           [0.0, 0.1, 3.0, -1.0, 2.0, 2.5, -1.0]], device=DEV)
    t, n, top, ns = 3, 6, 3, 2
    tiles = k.max_tiles(t, top + ns, n + ns)
    pairs = t * (top + ns)
    idx, place, order = (torch.zeros(pairs, dtype=torch.int32, device=DEV) for _ in range(3))
    weight, gate = torch.zeros(pairs, device=DEV), torch.zeros(t, device=DEV)
    count = torch.zeros(n + ns, dtype=torch.int32, device=DEV)
    plan = torch.zeros(k.plan_ints(n + ns, tiles), dtype=torch.int32, device=DEV)
    k.route(logits, top, idx, weight, place, count, plan, tiles, order, n_experts=n, groups=(3, 2), n_shared=ns,
            gate_col=n, scale=0.5, gate_out=gate)
    assert idx.view(t, -1).tolist() == [[0, 4, 5, 6, 7], [0, 1, 2, 6, 7], [2, 5, 4, 6, 7]]
    g = 0.5 * torch.sigmoid(logits[:, n]).cpu()
    assert torch.allclose(gate.cpu(), g)
    wt = weight.view(t, -1).cpu()
    assert torch.allclose(wt[:, 3], g) and torch.allclose(wt[:, 4], g)
    for i, chosen in enumerate([[0, 4, 5], [0, 1, 2], [2, 5, 4]]):
        assert torch.allclose(wt[i, :3], 0.5 * torch.softmax(logits[i, chosen].cpu(), -1))
    assert count.tolist() == [0] * (n + ns) and sorted(order.tolist()) == list(range(pairs))
    for bad in ({"groups": (4, 2)}, {"groups": (3, 1)}, {"groups": (3, 4)}):
        with pytest.raises(k.KernelError):
            k.route(logits, top, idx, weight, place, count, plan, tiles, order, n_experts=n, **bad)
