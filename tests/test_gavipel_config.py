"""The Gavipel design without a GPU: its config reader and the errors it gives, the run order of a
repeated run that is entered through a matrix, tensor names and shapes, storage planning, the
stretched rotation, the random folder, and the plain model's own rules."""
import copy
import math

import pytest
import torch

import gavipel_cases as cases
import helpers
import plain_gavipel as plain
from crucible_b200.config.model_config import ConfigError, FeedForwardSpec, PositionSpec
from crucible_b200.config.registry import known_architectures, parse_config
from crucible_b200.models.decoder import DecoderModel
from crucible_b200.parts import ARRANGEMENTS, FEED_FORWARDS, POSITIONS


def _config(name="ga-a"):
    return copy.deepcopy(cases.CASES[name]["config"])


def test_the_architecture_is_registered_and_parsed():
    assert "Gavipel" in known_architectures()
    cfg = parse_config(_config())
    assert (cfg.vocab_size, cfg.hidden_size, cfg.tie_word_embeddings) == (300, 64, True)
    assert [(layer.arrangement, layer.mixer.kind, layer.feed_forward.kind) for layer in cfg.layers] == \
        [("parallel_two_norms", "sink_attention", kind) for kind in ("moe", "moe", "none", "moe", "moe")]
    assert all(layer.option("layer_scale") is True and all(n.kind == "rmsnorm_offset" and n.eps == 1e-6 for _, n in layer.norms)
               for layer in cfg.layers)
    assert [[name for name, _ in layer.norms] for layer in cfg.layers[1:3]] == [["mixer_norm", "feed_forward_norm"], ["mixer_norm"]]
    a = cfg.layers[0].mixer
    assert (a.n_heads, a.n_kv_heads, a.head_dim, a.option("value_dim"), a.softmax_scale, a.window, a.option("sink"),
            a.option("gate"), a.option("qk_norm_eps"), a.option("value_norm_eps"), a.option("keep_first")) == \
        (4, 2, 16, 24, 0.4, 21, 0.0, "element", 1e-6, None, 0)
    assert not isinstance(a.option("sink"), bool)
    assert (a.position.kind, a.position.rotary_dim, a.position.theta, dict(a.position.scaling)) == \
        ("rope_interleaved", 8, 1000.0, {"factor": 8.0, "low": 1.0, "high": 3.0, "original": 40.0})
    assert cfg.layers[1].mixer.position.scaling is None and cfg.layers[3].mixer.position is None
    assert cfg.layers[2].mixer.window is None
    f = cfg.layers[0].feed_forward
    assert (f.intermediate, f.option("experts"), f.option("top"), f.option("groups"), f.option("score"),
            f.option("group_score"), f.option("shared_intermediate")) == (24, 6, 2, (3, 2), "sigmoid", "two_best", 40)
    assert cfg.layers[3].feed_forward.option("groups") is None
    assert cfg.layers[4].feed_forward.option("shared_intermediate") is None
    assert cfg.embedding.option("scale") == 7.3 and cfg.head.kind == "linear"
    # layers 1..3 twice, each pass entered through the matrix
    assert [(e.layer, e.copy, e.project, e.add, e.add_embedding) for e in cfg.run_order] == [
        (0, 0, None, None, False), (1, 0, "loop_in", None, False), (2, 0, None, None, False), (3, 0, None, None, False),
        (1, 1, "loop_in", None, False), (2, 1, None, None, False), (3, 1, None, None, False), (4, 0, None, None, False)]
    assert cfg.matrices == ("loop_in",) and cfg.vectors == ()


def test_options_that_are_absent():
    cfg = parse_config(_config("ga-d"))
    assert [(e.layer, e.copy, e.project) for e in cfg.run_order] == [(i, 0, None) for i in range(3)]
    assert cfg.matrices == ()
    raw = _config()
    raw["layers"][0]["mixer"].pop("kv_heads")
    raw["layers"][0]["mixer"].pop("vdim")
    raw["layers"][0]["mixer"]["rot"].pop("dims")
    raw["layers"][1]["mixer"]["rot"]["dims"] = 0
    raw.pop("embedding")
    cfg = parse_config(raw)
    assert (cfg.layers[0].mixer.n_kv_heads, cfg.layers[0].mixer.option("value_dim")) == (4, 16)
    assert cfg.layers[0].mixer.position.rotary_dim == 16 and cfg.layers[1].mixer.position is None
    assert cfg.embedding.option("scale") == 1.0
    empty = _config()
    empty["loop"].update(start=2, stop=2, times=3)
    assert [(e.layer, e.project) for e in parse_config(empty).run_order] == [(i, None) for i in range(5)]
    once = _config()
    once["loop"]["times"] = 1
    assert [(e.layer, e.project) for e in parse_config(once).run_order] == \
        [(0, None), (1, "loop_in"), (2, None), (3, None), (4, None)]


@pytest.mark.parametrize("edit,word", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mixer"].pop("heads"), "heads"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("original"), "original"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(high=0.5), "high"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "count"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=1), "keep"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["layers"][0].update(mlp=[1]), "mlp"),
    (lambda c: c["loop"].update(stop=9), "stop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["embedding"].update(scale="a"), "scale"),
    (lambda c: c.pop("layers"), "layers"),
])
def test_config_errors_name_the_key(edit, word):
    config = _config()
    edit(config)
    with pytest.raises(ConfigError) as e:
        parse_config(config)
    assert word in str(e.value)


def test_a_run_order_names_matrices_the_model_holds():
    import dataclasses
    cfg = parse_config(_config())
    with pytest.raises(ConfigError, match="loop_in"):
        dataclasses.replace(cfg, matrices=()).validate()


def test_tensor_names_shapes_and_storage():
    model = DecoderModel(parse_config(_config()))
    shapes = {r.checkpoint_name: tuple(r.decl.shape) for r in model.tensor_requests()}
    assert shapes["embed"] == (300, 64) and "head" not in shapes and shapes["loop.in"] == (64, 128)
    assert shapes["final.norm"] == (64,) and shapes["l0.norm1"] == (64,) and shapes["l0.norm2"] == (64,)
    assert shapes["l0.ls1"] == (64,) and shapes["l0.ls2"] == (64,)
    assert "l2.norm2" not in shapes and "l2.ls2" not in shapes and shapes["l2.ls1"] == (64,)
    assert shapes["l0.mix.q"] == (64, 64) and shapes["l0.mix.k"] == (32, 64) and shapes["l0.mix.v"] == (48, 64)
    assert shapes["l0.mix.g"] == (96, 64) and shapes["l0.mix.o"] == (64, 96) and "l0.mix.sink" not in shapes
    assert shapes["l0.mix.q.norm"] == (16,) and shapes["l0.mix.k.norm"] == (16,)
    assert shapes["l0.mlp.router"] == (6, 64) and shapes["l0.mlp.correction"] == (6,)
    assert shapes["l0.mlp.e5.down"] == (64, 24) and shapes["l0.mlp.shared.up"] == (40, 64)
    assert "l0.mlp.shared.sg" not in shapes and "l4.mlp.shared.up" not in shapes
    # layers of equal needs share pages; every pass has a slot of its own
    needs = {(g.need.head_dim, g.need.window): g.layers for g in model.cache_groups}
    assert needs == {(16, 21): (0, 4), (16, 40): (1, 1), (24, None): (2, 2), (32, 9): (3, 3)}
    assert model.state_bytes == 0
    assert [model.bindings[i].slot for i in (1, 4)] == [0, 1]
    assert "loop.in" not in {r.checkpoint_name for r in DecoderModel(parse_config(_config("ga-d"))).tensor_requests()}


def test_the_random_folder_is_read_back_by_the_plain_model(tmp_path):
    for name in sorted(cases.CASES):
        folder = cases.make_folder(tmp_path, name)
        config, tensors = plain.load_folder(folder)
        assert config["architecture"] == "Gavipel"
        model = DecoderModel(parse_config(config))
        assert {r.checkpoint_name: tuple(r.decl.shape) for r in model.tensor_requests()} == \
            {k: tuple(v.shape) for k, v in tensors.items()}
        logits = plain.forward(config, tensors, [1, 2, 3, 4, 5])
        assert tuple(logits.shape) == (5, config["vocab"]) and bool(torch.isfinite(logits).all())


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_the_cases_leave_no_close_call_to_a_router(tmp_path, name, monkeypatch):
    folder = cases.make_folder(tmp_path, name)
    config, tensors = plain.load_folder(folder)
    least, chosen, real = [], set(), plain.choose_experts

    def watched(choice, top, groups, keep):
        least.append(cases.margin(choice.tolist(), top, groups, keep))
        out = real(choice, top, groups, keep)
        chosen.add(tuple(out))
        return out
    monkeypatch.setattr(plain, "choose_experts", watched)
    plain.forward(config, tensors, helpers.random_tokens(config["vocab"], 60, 1))
    assert min(least) > 0.02 and len(chosen) > 3


# ---- the stretched rotation --------------------------------------------------------------------

@pytest.mark.parametrize("dims,base,scaling", [
    (64, 10000.0, (8.0, 1.0, 4.0, 512.0)), (48, 500000.0, (32.0, 2.0, 3.0, 4096.0)), (6, 10.0, (2.0, 1.0, 1.0, 20.0)),
    (10, 50.0, None), (2, 50.0, (2.0, 1.0, 4.0, 20.0))])
def test_stretched_frequencies(dims, base, scaling):
    named = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    part = POSITIONS.build("rope_interleaved", PositionSpec("rope_interleaved", dims, base, 0,
                                                            tuple(named.items()) if named else None))
    part.bind({}, torch.bfloat16, torch.device("cpu"))
    freq, n = part.frequencies()
    want = plain.turning_rates(dims, base, named)
    assert n == dims and freq.dtype == torch.float32
    assert torch.equal(freq, want.to(torch.float32))
    if dims == 64:
        # all three ranges are there: as they are, slowed down, and between
        ratio = want / plain.turning_rates(dims, base)
        assert int((ratio == 1.0).sum()) > 2 and int((ratio - 1 / 8).abs().lt(1e-12).sum()) > 2
        assert int(((ratio < 0.999) & (ratio > 0.126)).sum()) > 2
    with pytest.raises(ValueError):
        POSITIONS.build("rope_interleaved", PositionSpec("rope_interleaved", 8, 10.0, 0, (("factor", 2.0),)))


# ---- parts that refuse ------------------------------------------------------------------------------

def test_parts_refuse_what_they_cannot_do():
    spec = parse_config(_config()).layers[0]
    model = DecoderModel(parse_config(_config()))
    layer = model.layers[0]
    swiglu = FEED_FORWARDS.build("swiglu", FeedForwardSpec(kind="swiglu", width=64, intermediate=32))
    with pytest.raises(ValueError, match="open"):
        ARRANGEMENTS.build("parallel_two_norms", spec, layer.norms, layer.mixer, swiglu)

    class Adds:
        pass
    with pytest.raises(ValueError, match="write"):
        ARRANGEMENTS.build("parallel_two_norms", spec, layer.norms, Adds(), layer.feed_forward)
    for extra in ((("score", "max"),), (("group_score", "mean"),)):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build("moe", FeedForwardSpec(kind="moe", width=8, intermediate=8,
                                                       extra=(("experts", 4), ("top", 1)) + extra))


# ---- the plain model's own rules -------------------------------------------------------------

def test_plain_run_list_and_entry():
    config = {"layers": [0, 1, 2, 3], "loop": {"start": 1, "stop": 3, "times": 2}}
    assert plain.run_list(config) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    w = torch.randn(3, 6, dtype=torch.float64)
    x, x0 = torch.randn(2, 3, dtype=torch.float64), torch.randn(2, 3, dtype=torch.float64)
    assert torch.allclose(plain.enter_pass(x, x0, w), x @ w[:, :3].T + x0 @ w[:, 3:].T)


def test_plain_window_and_softmax():
    assert [row.nonzero().flatten().tolist() for row in plain.seen_in_window(5, 2)] == [[0], [0, 1], [1, 2], [2, 3], [3, 4]]
    assert bool(plain.seen_in_window(4).equal(torch.ones(4, 4, dtype=torch.bool).tril()))
    p = plain.softmax_plus_one(torch.tensor([[1.0, -2.0, 50.0]]).double(), torch.tensor([[True, True, False]]))
    total = 1.0 + math.exp(1.0) + math.exp(-2.0)
    assert torch.allclose(p, torch.tensor([[math.exp(1.0) / total, math.exp(-2.0) / total, 0.0]]).double())
    far = plain.softmax_plus_one(torch.tensor([[-800.0]]).double(), torch.tensor([[True]]))
    assert float(far) == 0.0


def test_plain_choice_of_experts():
    # groups (0, 1) (2, 3) (4, 5): the best single score is in the first, the best sum in the second
    c = torch.tensor([0.9, -0.8, 0.5, 0.4, 0.3, 0.2])
    assert plain.choose_experts(c, 2, 3, 1) == [2, 3]
    assert plain.choose_experts(c, 2, 3, 2) == [2, 3]                # (0.5 + 0.4, 0.3 + 0.2)
    assert plain.choose_experts(c, 2, 1, 1) == [0, 2]
    # all scores negative: what is left out counts as minus infinity, not as zero
    assert plain.choose_experts(c - 2.0, 2, 3, 1) == [2, 3]
    # groups of one expert: a group's score is that expert's
    assert plain.choose_experts(c, 2, 6, 2) == [0, 2]
    # the weights are the scores without the correction, as they are
    w = {"router": torch.tensor([[0.0], [0.0]]), "correction": torch.tensor([5.0, 1.0])}
    for e, value in ((0, 2.0), (1, 3.0)):
        w.update({f"e{e}.gate": torch.tensor([[30.0]]), f"e{e}.up": torch.tensor([[1.0]]),
                  f"e{e}.down": torch.tensor([[value / 30.0]])})
    out = plain.mixture(torch.ones(1, 1).double(), {k: v.double() for k, v in w.items()},
                        {"router": {"experts": 2, "top": 1}}, "")
    assert abs(float(out) - 0.5 * 2.0) < 1e-6
