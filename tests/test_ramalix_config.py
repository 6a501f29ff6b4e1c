"""The Ramalix design without a GPU: its config reader and the errors it gives, the run order of
a repeated run that takes the embedding again, tensor names and shapes, storage planning (slots,
states and convolution inputs for every pass), pages given back chunk by chunk, the random folder,
and the plain model's own rules."""
import copy
import math

import pytest
import torch

import plain_ramalix as plain
import ramalix_cases as cases
from crucible_b200.cache import CacheManager, GroupPolicy
from crucible_b200.config.model_config import ConfigError
from crucible_b200.config.registry import known_architectures, parse_config
from crucible_b200.models.decoder import DecoderModel


def _config(name="ra-a"):
    return copy.deepcopy(cases.CASES[name]["config"])


def test_the_architecture_is_registered_and_parsed():
    assert "Ramalix" in known_architectures()
    cfg = parse_config(_config())
    assert (cfg.vocab_size, cfg.hidden_size, cfg.tie_word_embeddings) == (300, 64, False)
    kinds = [(layer.arrangement, layer.mixer.kind, layer.feed_forward.kind) for layer in cfg.layers]
    assert kinds == [("pre_norm_conv", "channel_delta", "moe"), ("pre_norm_conv", "differential_attention", "moe"),
                     ("pre_norm_conv", "sink_attention", "none"), ("pre_norm_conv", "channel_delta", "moe"),
                     ("pre_norm_conv", "sink_attention", "moe")]
    assert all(layer.option("taps") == 4 and all(n.kind == "rmsnorm_one_number" for _, n in layer.norms)
               for layer in cfg.layers)
    assert [name for name, _ in cfg.layers[2].norms] == ["mixer_norm"]
    d = cfg.layers[0].mixer
    assert (d.n_heads, d.n_kv_heads, d.head_dim, d.option("value_dim"), d.option("conv_taps"),
            d.option("out_scale")) == (4, 2, 16, 24, 4, 0.7)
    a = cfg.layers[1].mixer
    assert (a.n_heads, a.n_kv_heads, a.head_dim, a.option("value_dim"), a.softmax_scale, a.option("diff"),
            a.option("q_temp"), a.position) == (4, 2, 16, 24, 0.5, 0.3, (0.2, 10), None)
    c = cfg.layers[2].mixer
    assert (c.window, c.option("chunked"), c.option("sink"), c.option("gate"), c.option("value_norm_eps")) == \
        (21, True, True, None, None)
    assert (c.position.kind, c.position.rotary_dim, c.position.theta) == ("rope_interleaved", 8, 1000.0)
    f = cfg.layers[0].feed_forward
    assert (f.intermediate, f.option("experts"), f.option("top"), f.option("groups"), f.option("shared_intermediate"),
            f.option("shared_gate"), f.option("out_scale")) == (24, 6, 2, (3, 2), 40, True, 0.7)
    assert cfg.layers[4].feed_forward.option("shared_gate") is False
    assert cfg.head.option("scale") == 1.5 and cfg.embedding.kind == "token"
    # layers 1..3 twice: the embedding joins before the second pass alone, the passes' vectors before both
    assert [(e.layer, e.copy, e.add, e.add_embedding) for e in cfg.run_order] == [
        (0, 0, None, False), (1, 0, ("loop_step", 0), False), (2, 0, None, False), (3, 0, None, False),
        (1, 1, ("loop_step", 1), True), (2, 1, None, False), (3, 1, None, False), (4, 0, None, False)]
    assert cfg.vectors == (("loop_step", 2),)


def test_options_that_are_absent():
    cfg = parse_config(_config("ra-d"))
    assert [(e.layer, e.copy, e.add) for e in cfg.run_order] == [(i, 0, None) for i in range(4)]
    assert cfg.vectors == ()
    b = parse_config(_config("ra-b"))
    assert b.layers[0].mixer.position is None and b.layers[2].mixer.option("q_temp") is None
    assert b.layers[0].feed_forward.option("groups") is None
    raw = _config()
    raw["layers"][1]["mixer"].pop("kv_heads")
    raw["layers"][2]["mixer"].pop("mask")
    cfg = parse_config(raw)
    assert cfg.layers[1].mixer.n_kv_heads == 4
    assert cfg.layers[2].mixer.window is None and cfg.layers[2].mixer.option("chunked") is False
    empty = _config()
    empty["loop"].update(start=2, stop=2, times=3)
    cfg = parse_config(empty)
    assert [(e.layer, e.add, e.add_embedding) for e in cfg.run_order] == [(i, None, False) for i in range(5)]


@pytest.mark.parametrize("edit,word", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].pop("every"), "every"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(coef="x"), "coef"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "count"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=1), "keep"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["loop"].update(stop=9), "stop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.pop("canon"), "canon"),
    (lambda c: c.update(residual_mult="a"), "residual_mult"),
    (lambda c: c.update(logit_scale=None, residual_mult=float("nan")), "residual_mult"),
    (lambda c: c.pop("layers"), "layers"),
])
def test_config_errors_name_the_key(edit, word):
    config = _config()
    edit(config)
    with pytest.raises(ConfigError) as e:
        parse_config(config)
    assert word in str(e.value)


def test_tensor_names_shapes_and_storage():
    model = DecoderModel(parse_config(_config()))
    shapes = {r.checkpoint_name: tuple(r.decl.shape) for r in model.tensor_requests()}
    assert shapes["embed"] == (300, 64) and shapes["head"] == (300, 64)
    assert shapes["final.norm"] == () and shapes["l0.norm1"] == () and shapes["l0.norm2"] == ()
    assert "l2.norm2" not in shapes and "l2.canon2" not in shapes and shapes["l2.canon1"] == (64, 4)
    assert shapes["l0.canon1"] == (64, 4) and shapes["l0.canon2"] == (64, 4) and shapes["loop.step"] == (2, 64)
    assert shapes["l1.mix.q"] == (128, 64) and shapes["l1.mix.k"] == (64, 64) and shapes["l1.mix.v"] == (48, 64)
    assert shapes["l1.mix.q.b"] == (128,) and shapes["l1.mix.o.b"] == (64,) and shapes["l1.mix.lq2"] == (16,)
    assert shapes["l2.mix.sink"] == (4,) and shapes["l2.mix.o"] == (64, 96) and "l2.mix.g" not in shapes
    assert shapes["l0.mix.q"] == (32, 64) and shapes["l0.mix.v"] == (96, 64) and shapes["l0.mix.v.conv"] == (96, 4)
    assert shapes["l0.mix.dt_bias"] == (64,) and shapes["l0.mix.A_log"] == (4,) and shapes["l0.mix.norm"] == (24,)
    assert shapes["l0.mix.a2"][0] == 64 and shapes["l0.mix.g2"][0] == 96
    assert shapes["l0.mlp.router"] == (6, 64) and shapes["l0.mlp.shared.up"] == (40, 64)
    assert shapes["l0.mlp.shared.sg"] == (1, 64) and "l4.mlp.shared.sg" not in shapes
    # chunked layers share pages with no other layer; every pass has a slot
    needs = {(g.need.head_dim, g.need.window, g.need.chunked): g.layers for g in model.cache_groups}
    assert needs == {(32, None, False): (1, 1), (16, 21, True): (2, 2), (32, 40, True): (4,)}
    # every run has the inputs of its convolutions, beside a mixer's state, and no two overlap
    spans = []
    for entry, b in zip(model.config.run_order, model.bindings):
        layer = model.layers[entry.layer]
        assert b.own.state_bytes == (2 if layer.has_ffn else 1) * 4 * 3 * 64
        spans.append((b.own.state_offset, b.own.state_bytes))
        if b.state_bytes:
            spans.append((b.state_offset, b.state_bytes))
    ends = sorted((o, o + n) for o, n in spans)
    assert all(a[1] <= b[0] for a, b in zip(ends, ends[1:])) and ends[-1][1] <= model.state_bytes
    assert len(spans) == 8 + 3
    # one tap: nothing to remember
    assert all(b.own is None for b in DecoderModel(parse_config(_config("ra-d"))).bindings)


def test_chunks_give_their_pages_back():
    """A group with chunks of 10 over pages of 4: what lies wholly before the chunk of the next
    token goes back, and no page a chunk still needs."""
    m = CacheManager([GroupPolicy(4, window=10, chunked=True), GroupPolicy(4)], [40, 40], n_state_slots=2,
                     table_strides=[40, 40], null_pages=[40, 40])
    m.add_request("a")
    length = 0
    for n in [3, 1, 5, 1, 1, 9, 2, 20, 1, 1, 30, 7]:
        m.extend("a", n)
        first_needed = length // 10 * 10           # of the step's first token
        table = m.block_table("a", 0)
        length += n
        assert len(table) == -(-length // 4)
        assert [p >= 0 for p in table] == [b >= first_needed // 4 for b in range(len(table))]
        assert all(p >= 0 for p in m.block_table("a", 1))
        m.check_invariants()
    # what a request of 200 tokens in steps of 5 holds at most: a chunk less one, a step, the edges
    assert m.pages_for(0, 200, 5) == -(-(9 + 5) // 4) + 1
    m.remove_request("a")
    assert m.free_pages(0) == 40
    with pytest.raises(ValueError):
        CacheManager([GroupPolicy(4, chunked=True)], [4], n_state_slots=1)


def test_the_random_folder_is_read_back_by_the_plain_model(tmp_path):
    for name in sorted(cases.CASES):
        folder = cases.make_folder(tmp_path, name)
        config, tensors = plain.load_folder(folder)
        assert config["architecture"] == "Ramalix"
        model = DecoderModel(parse_config(config))
        assert {r.checkpoint_name: tuple(r.decl.shape) for r in model.tensor_requests()} == \
            {k: tuple(v.shape) for k, v in tensors.items()}
        logits = plain.forward(config, tensors, [1, 2, 3, 4, 5])
        assert tuple(logits.shape) == (5, config["vocab"]) and bool(torch.isfinite(logits).all())


# ---- the plain model's own rules -------------------------------------------------------------

def test_plain_run_list():
    config = {"layers": [0, 1, 2, 3], "loop": {"start": 1, "stop": 3, "times": 3}}
    assert plain.run_list(config) == [(0, None, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False),
                                      (1, 2, True), (2, 2, False), (3, None, False)]


def test_plain_convolution_and_chunks():
    x = torch.randn(6, 2, dtype=torch.float64)
    w = torch.randn(2, 3, dtype=torch.float64)
    y = plain.causal_conv(x, w)
    for t in range(6):
        want = sum(w[:, j] * x[t - 2 + j] for j in range(3) if t - 2 + j >= 0)
        assert torch.allclose(y[t], want)
    assert torch.allclose(plain.input_conv(x, w), x + y)
    seen = plain.seen_in_chunk(7, 3)
    assert [row.nonzero().flatten().tolist() for row in seen] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]


def test_plain_temperature_sink_and_groups():
    t = plain.query_temperature(torch.arange(12), 0.5, 5, torch.float64)
    want = [1.0] * 4 + [1 + 0.5 * math.log(2)] * 5 + [1 + 0.5 * math.log(3)] * 3
    assert torch.allclose(t, torch.tensor(want, dtype=torch.float64))
    p = plain.softmax_over(torch.tensor([[[1.0]]]).double(), torch.ones(1, 1, dtype=torch.bool), torch.tensor([1.5]).double())
    assert abs(float(p) - math.exp(1.0) / (math.exp(1.0) + math.exp(1.5))) < 1e-12
    # the best experts overall are 0 and 1; with one kept group of two the second best is expert 1
    s = torch.tensor([0.4, 0.05, 0.3, 0.25])
    assert plain.choose_experts(s, 2, 1, 1) == [0, 2]
    assert plain.choose_experts(s, 2, 2, 1) == [0, 1]
    assert plain.choose_experts(s, 2, 4, 3) == [0, 2]


def test_plain_delta_rule_overwrites_and_forgets():
    """With beta near 1 and one unit key the state answers with the key's last value; a channel
    whose decay is near 0 forgets what the others keep."""
    g = torch.Generator().manual_seed(0)
    W, D, E, t = 6, 4, 3, 5
    w = {"q": torch.randn(D, W, generator=g), "k": torch.randn(D, W, generator=g), "v": torch.randn(E, W, generator=g),
         "q.conv": torch.tensor([[1.0]] * D), "k.conv": torch.tensor([[1.0]] * D), "v.conv": torch.tensor([[1.0]] * E),
         "b": torch.zeros(1, W), "A_log": torch.zeros(1), "a1": torch.randn(2, W, generator=g), "a2": torch.zeros(D, 2),
         "dt_bias": torch.tensor([-30.0, -30.0, 30.0, -30.0]), "norm": torch.ones(E), "g1": torch.zeros(2, W),
         "g2": torch.zeros(E, 2), "o": torch.randn(W, E, generator=g)}
    w = {k: v.double() for k, v in w.items()}
    # channel 2 holds the last token's write alone, the others those of all tokens
    h = torch.randn(t, W, generator=torch.Generator().manual_seed(1)).double()
    states = []
    plain.channel_delta(h, w, {"heads": 1, "dim": D, "vdim": E}, 1e-6, "", states)
    k = plain.silu(h @ w["k"].T)
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    v = plain.silu(h @ w["v"].T)
    S = torch.zeros(D, E, dtype=torch.float64)
    keep = torch.tensor([1.0, 1.0, math.exp(-30.0), 1.0]).double()
    for i in range(t):
        S = keep[:, None] * S
        S = S + 0.5 * k[i][:, None] * (v[i] - S.T @ k[i])[None, :]
    assert torch.allclose(states[0][0], S, atol=1e-9)
