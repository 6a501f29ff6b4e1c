"""Gavipel: a decoder whose layers are listed one by one in config.json; the two sublayers of a
layer read the same residual through a norm each and are scaled element by element,
x += ls1 * mixer(norm1(x)) + ls2 * ff(norm2(x)); every such norm's weight is stored around zero (the
gain is 1 + weight); a run of layers may repeat with the same weights.

config.json: `vocab`, `width`, `norm.eps`, `embedding.scale`, `layers` (a list of {`type`, `mixer`,
`mlp`}) and `loop` = {`start`, `stop`, `times`}: the layers start .. stop - 1 run `times` times in a
row, each pass with keys of its own; before every pass x becomes `loop.in` [x; embedding's output],
`loop.in` [width, 2 width].  One layer type:
  `attention`: grouped-query attention (`heads`, `kv_heads`, `dim`, `vdim`, `scale`) with an RMS
      norm of every q and k head (one weight over `dim` for all heads, stored as the gain itself),
      the rotation of neighbouring pairs on the first `rot.dims` features (`rot.base`, and
      `rot.scaling` = {`factor`, `low`, `high`, `original`} or absent), a window of `mask.size`
      keys (absent: all earlier ones), one more in the softmax's denominator, and a sigmoid gate
      with a logit for every output feature.
`mlp` is null or {`kind`: "moe", `router`: {`experts`, `top`, `groups`: {`count`, `keep`} or absent},
`expert`: {`ff`}, `shared`: {`ff`} or absent}: experts are chosen by sigmoid(logit) + `correction`
from the groups whose two best have the largest sum, and weighted by sigmoid(logit) as it is.
The head is the embedding's table, without the scale.  Tensors: `embed`, `loop.in`, `final.norm`, and
per layer `l<i>.norm1|norm2`, `l<i>.ls1|ls2`, `l<i>.mix.*`, `l<i>.mlp.*`.  The design names no longest
context.
"""
from __future__ import annotations

import copy
from collections.abc import Mapping as _Mapping
from typing import Any, Mapping

from ..config.model_config import (UNBOUNDED_CONTEXT, ConfigError, EndSpec, FeedForwardSpec, KeyReader,
                                   LayerSpec, MixerSpec, ModelConfig, NormSpec, PositionSpec)
from ..config.registry import Architecture, register_architecture
from .loops import LOOP_MATRIX, looped_run_order

# the score of the softmax's sink, fixed by the design: exp(0) = 1 joins the denominator
SINK_SCORE = 0.0


class _Names(_Mapping):
    """Part-local tensor names to this family's checkpoint names, by rule."""
    _FIXED = {"embedding.table": "embed", "final_norm.gain": "final.norm",
              "layer.mixer_norm.gain": "l{layer}.norm1", "layer.feed_forward_norm.gain": "l{layer}.norm2",
              "layer.arrangement.mixer_scale": "l{layer}.ls1",
              "layer.arrangement.feed_forward_scale": "l{layer}.ls2", f"matrices.{LOOP_MATRIX}": "loop.in"}
    _PREFIXES = (("layer.mixer.", "l{layer}.mix."), ("layer.feed_forward.", "l{layer}.mlp."))

    def __getitem__(self, key):
        if key in self._FIXED:
            return self._FIXED[key]
        for local, stored in self._PREFIXES:
            if key.startswith(local):
                return stored + key[len(local):]
        raise KeyError(key)

    def __iter__(self):
        return iter(self._FIXED)

    def __len__(self):
        return len(self._FIXED)


def _section(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: {key!r} must be an object")
    return v


def _rotation(raw, dim: int, where: str):
    if raw.get("rot") is None:
        return None
    where += ".rot"
    rot = KeyReader(_section(raw, "rot", where), where)
    dims = rot.raw.get("dims", dim)
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"{where}: 'dims' must be even and at most {dim}, got {dims!r}")
    if dims == 0:
        return None
    scaling = None
    if rot.raw.get("scaling") is not None:
        s = KeyReader(_section(rot.raw, "scaling", where), where + ".scaling")
        scaling = tuple((key, s.number(key)) for key in ("factor", "low", "high", "original"))
        if dict(scaling)["high"] < dict(scaling)["low"]:
            raise ConfigError(f"{where}.scaling: 'high' must not be below 'low'")
    return PositionSpec(kind="rope_interleaved", rotary_dim=dims, theta=rot.number("base"), max_positions=0,
                        scaling=scaling)


def _attention(raw, width: int, eps: float, where: str) -> MixerSpec:
    r = KeyReader(raw, where)
    dim, heads = r.integer("dim"), r.integer("heads")
    kv_heads = r.integer("kv_heads", heads)
    if heads % kv_heads:
        raise ConfigError(f"{where}: 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    window = None
    if raw.get("mask") is not None:
        window = KeyReader(_section(raw, "mask", where), where + ".mask").integer("size")
    return MixerSpec(kind="sink_attention", width=width, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim,
                     softmax_scale=r.number("scale"), window=window, position=_rotation(raw, dim, where),
                     extra=(("value_dim", r.integer("vdim", dim)), ("keep_first", 0), ("sink", SINK_SCORE),
                            ("gate", "element"), ("value_norm_eps", None), ("qk_norm_eps", eps)))


_MIXERS = {"attention": _attention}


def _feed_forward(mlp, width: int, where: str) -> FeedForwardSpec:
    if mlp is None:
        return FeedForwardSpec(kind="none", width=width, intermediate=0)
    if not isinstance(mlp, dict):
        raise ConfigError(f"{where}: 'mlp' must be an object or null")
    KeyReader(mlp, where).choice("kind", ("moe",))
    router = KeyReader(_section(mlp, "router", where), where + ".router")
    experts, top = router.integer("experts"), router.integer("top")
    if top > experts:
        raise ConfigError(f"{where}.router: 'top' ({top}) exceeds 'experts' ({experts})")
    groups = None
    if mlp["router"].get("groups") is not None:
        g = KeyReader(_section(mlp["router"], "groups", where + ".router"), where + ".router.groups")
        count, keep = g.integer("count"), g.integer("keep")
        if experts % count or keep > count or top > keep * (experts // count):
            raise ConfigError(f"{where}.router.groups: 'count' ({count}) must divide the experts ({experts}), 'keep' "
                              f"({keep}) be at most 'count', and the kept groups hold at least 'top' ({top}) experts")
        groups = (count, keep)
    shared = None
    if mlp.get("shared") is not None:
        shared = KeyReader(_section(mlp, "shared", where), where + ".shared").integer("ff")
    return FeedForwardSpec(kind="moe", width=width,
                           intermediate=KeyReader(_section(mlp, "expert", where), where + ".expert").integer("ff"),
                           extra=(("experts", experts), ("top", top), ("groups", groups), ("score", "sigmoid"),
                                  ("group_score", "two_best"), ("shared_intermediate", shared), ("open_sum", True)))


def _parse(raw: Mapping[str, Any]) -> ModelConfig:
    r = KeyReader(raw)
    width, vocab = r.integer("width"), r.integer("vocab")
    eps = KeyReader(_section(raw, "norm", "config.json"), "config.json norm").number("eps")
    scale = 1.0
    if raw.get("embedding") is not None:
        scale = KeyReader(_section(raw, "embedding", "config.json"), "config.json embedding").number("scale", 1.0)
    entries = raw.get("layers")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config.json: 'layers' must be a list with at least one layer")
    norm = NormSpec(kind="rmsnorm_offset", width=width, eps=eps)
    layers = []
    for i, entry in enumerate(entries):
        where = f"config.json layers[{i}]"
        if not isinstance(entry, dict) or not isinstance(entry.get("type"), str):
            raise ConfigError(f"{where}: a layer is an object with a 'type'")
        kind = entry["type"]
        if kind not in _MIXERS:
            raise ConfigError(f"{where}: unknown layer type {kind!r} (this engine runs {sorted(_MIXERS)})")
        mixer = _MIXERS[kind](_section(entry, "mixer", where), width, eps, where + ".mixer")
        ffn = _feed_forward(entry.get("mlp"), width, where + ".mlp")
        norms = (("mixer_norm", norm),) + ((("feed_forward_norm", norm),) if ffn.kind != "none" else ())
        layers.append(LayerSpec(arrangement="parallel_two_norms", mixer=mixer, feed_forward=ffn, norms=norms,
                                extra=(("layer_scale", True),)))
    order, times = looped_run_order(raw, len(layers), project=True)
    return ModelConfig(
        architecture="Gavipel", vocab_size=vocab, hidden_size=width, max_context=UNBOUNDED_CONTEXT,
        tie_word_embeddings=True, layers=tuple(layers), run_order=order, final_norm=norm,
        embedding=EndSpec("token_hashed_positions", (("scale", scale), ("bigram", None), ("max_positions", None))),
        matrices=(LOOP_MATRIX,) if times else (),
        tensor_names=_Names(), raw=copy.deepcopy(dict(raw)))


def _describe(cfg: ModelConfig) -> dict:
    out = copy.deepcopy(dict(cfg.raw))
    out["architecture"] = "Gavipel"
    return out


register_architecture(Architecture("Gavipel", _parse, _describe))
