"""Ramalix: a decoder whose layers are listed one by one in config.json; pre-norm layers whose
norms have ONE number as their gain, with a short causal convolution on what each sublayer reads
(x += m mixer(c1(norm1(x))); x += m ff(c2(norm2(x))), c(h)_t = h_t + sum_j w_j h_(t-taps+1+j)); a
run of layers may repeat with the same weights.

config.json: `vocab`, `width`, `norm.eps`, `residual_mult` (m), `logit_scale`, `canon.taps`,
`layers` (a list of {`type`, `mixer`, `mlp`}) and `loop` = {`start`, `stop`, `times`}: the layers
start .. stop - 1 run `times` times in a row, each pass with keys and state of its own; before each
pass but the first the embedding's output is added to the residual, then before each pass row t of
the tensor `loop.step` [times, width].  Layer types:
  `attention`: two softmax maps per head over the same values, a_1 - lambda a_2, normed per head
      (`heads`, `kv_heads`, `dim`, `vdim`, `scale`, `diff`, `q_temp` = {`coef`, `every`} or absent:
      q times 1 + coef ln(floor((p + 1) / every) + 1)); biases, no rotation;
  `attention_2`: grouped-query attention (`heads`, `kv_heads`, `dim`, `vdim`, `scale`) with the
      rotation of neighbouring pairs on the first `rot.dims` features (`rot.base`), keys of the
      row's own chunk of `mask.size` positions, and a learned sink per head;
  `channel_delta`: the delta rule with a decay per key channel (`heads`, `kv_heads`, `dim`, `vdim`,
      `conv`: taps of the short convolution), a sigmoid gate through a low rank.
`mlp` is null or {`kind`: "moe", `router`: {`experts`, `top`, `groups`: {`count`, `keep`} or absent},
`expert`: {`ff`}, `shared`: {`ff`} or absent (times the sigmoid of one logit a token)}.
Tensors: `embed`, `loop.step`, `final.norm` and `l<i>.norm1|norm2` (shape []), `head`, and per layer
`l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.canon1|canon2`.  The design names no longest context.
"""
from __future__ import annotations

import copy
import math
from collections.abc import Mapping as _Mapping
from typing import Any, Mapping, Optional

from ..config.model_config import (UNBOUNDED_CONTEXT, ConfigError, EndSpec, FeedForwardSpec, KeyReader,
                                   LayerSpec, MixerSpec, ModelConfig, NormSpec, PositionSpec)
from ..config.registry import Architecture, register_architecture
from .loops import LOOP_VECTORS, looped_run_order


class _Names(_Mapping):
    """Part-local tensor names to this family's checkpoint names, by rule."""
    _FIXED = {"embedding.table": "embed", "final_norm.gain": "final.norm", "head.weight": "head",
              "layer.mixer_norm.gain": "l{layer}.norm1", "layer.feed_forward_norm.gain": "l{layer}.norm2",
              "layer.arrangement.mixer_conv": "l{layer}.canon1",
              "layer.arrangement.feed_forward_conv": "l{layer}.canon2", f"vectors.{LOOP_VECTORS}": "loop.step"}
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


def _real(raw: Mapping[str, Any], key: str, where: str, default: Optional[float] = None) -> float:
    """A finite number of either sign."""
    v = raw.get(key)
    if v is None and default is not None:
        return default
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v):
        raise ConfigError(f"{where}: {key!r} must be a finite number, got {v!r}")
    return float(v)


def _heads(r: KeyReader, where: str):
    """(heads, kv_heads, dim, vdim)"""
    heads, dim = r.integer("heads"), r.integer("dim")
    kv_heads = r.integer("kv_heads", heads)
    if heads % kv_heads:
        raise ConfigError(f"{where}: 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    return heads, kv_heads, dim, r.integer("vdim", dim)


def _differential(raw, width: int, eps: float, mult: float, where: str) -> MixerSpec:
    r = KeyReader(raw, where)
    heads, kv_heads, dim, vdim = _heads(r, where)
    temp = None
    if raw.get("q_temp") is not None:
        q = _section(raw, "q_temp", where)
        temp = (_real(q, "coef", where + ".q_temp"), KeyReader(q, where + ".q_temp").integer("every"))
    return MixerSpec(kind="differential_attention", width=width, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim,
                     softmax_scale=r.number("scale"), window=None,
                     extra=(("value_dim", vdim), ("diff", _real(raw, "diff", where)), ("norm_eps", eps),
                            ("q_temp", temp), ("out_scale", mult)))


def _chunked(raw, width: int, eps: float, mult: float, where: str) -> MixerSpec:
    r = KeyReader(raw, where)
    heads, kv_heads, dim, vdim = _heads(r, where)
    position = None
    if raw.get("rot") is not None:
        rot = KeyReader(_section(raw, "rot", where), where + ".rot")
        dims = rot.raw.get("dims", dim)
        if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > dim:
            raise ConfigError(f"{where}.rot: 'dims' must be even and at most {dim}, got {dims!r}")
        if dims:
            position = PositionSpec(kind="rope_interleaved", rotary_dim=dims, theta=rot.number("base"),
                                    max_positions=0)
    size = None
    if raw.get("mask") is not None:
        size = KeyReader(_section(raw, "mask", where), where + ".mask").integer("size")
    return MixerSpec(kind="sink_attention", width=width, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim,
                     softmax_scale=r.number("scale"), window=size, position=position,
                     extra=(("value_dim", vdim), ("keep_first", 0), ("sink", True), ("gate", None),
                            ("value_norm_eps", None), ("qk_norm_eps", None), ("chunked", size is not None),
                            ("out_scale", mult)))


def _channel_delta(raw, width: int, eps: float, mult: float, where: str) -> MixerSpec:
    r = KeyReader(raw, where)
    heads, kv_heads, dim, vdim = _heads(r, where)
    return MixerSpec(kind="channel_delta", width=width, n_heads=heads, n_kv_heads=kv_heads, head_dim=dim,
                     extra=(("value_dim", vdim), ("conv_taps", r.integer("conv")), ("norm_eps", eps),
                            ("out_scale", mult)))


_MIXERS = {"attention": _differential, "attention_2": _chunked, "channel_delta": _channel_delta}


def _feed_forward(mlp, width: int, mult: float, where: str) -> FeedForwardSpec:
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
                           extra=(("experts", experts), ("top", top), ("groups", groups),
                                  ("shared_intermediate", shared), ("shared_gate", shared is not None),
                                  ("out_scale", mult)))


def _parse(raw: Mapping[str, Any]) -> ModelConfig:
    r = KeyReader(raw)
    width, vocab = r.integer("width"), r.integer("vocab")
    eps = KeyReader(_section(raw, "norm", "config.json"), "config.json norm").number("eps")
    taps = KeyReader(_section(raw, "canon", "config.json"), "config.json canon").integer("taps")
    mult = _real(raw, "residual_mult", "config.json", 1.0)
    entries = raw.get("layers")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config.json: 'layers' must be a list with at least one layer")
    norm = NormSpec(kind="rmsnorm_one_number", width=width, eps=eps)
    layers = []
    for i, entry in enumerate(entries):
        where = f"config.json layers[{i}]"
        if not isinstance(entry, dict) or not isinstance(entry.get("type"), str):
            raise ConfigError(f"{where}: a layer is an object with a 'type'")
        kind = entry["type"]
        if kind not in _MIXERS:
            raise ConfigError(f"{where}: unknown layer type {kind!r} (this engine runs {sorted(_MIXERS)})")
        mixer = _MIXERS[kind](_section(entry, "mixer", where), width, eps, mult, where + ".mixer")
        ffn = _feed_forward(entry.get("mlp"), width, mult, where + ".mlp")
        norms = (("mixer_norm", norm),) + ((("feed_forward_norm", norm),) if ffn.kind != "none" else ())
        layers.append(LayerSpec(arrangement="pre_norm_conv", mixer=mixer, feed_forward=ffn, norms=norms,
                                extra=(("taps", taps),)))
    order, times = looped_run_order(raw, len(layers), embedding_again=True)
    return ModelConfig(
        architecture="Ramalix", vocab_size=vocab, hidden_size=width, max_context=UNBOUNDED_CONTEXT,
        tie_word_embeddings=False, layers=tuple(layers), run_order=order, final_norm=norm,
        embedding=EndSpec("token"),
        head=EndSpec("linear", (("scale", _real(raw, "logit_scale", "config.json", 1.0)),)),
        vectors=((LOOP_VECTORS, times),) if times else (),
        tensor_names=_Names(), raw=copy.deepcopy(dict(raw)))


def _describe(cfg: ModelConfig) -> dict:
    out = copy.deepcopy(dict(cfg.raw))
    out["architecture"] = "Ramalix"
    return out


register_architecture(Architecture("Ramalix", _parse, _describe))
