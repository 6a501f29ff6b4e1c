"""The generic decoder: embedding, a list of layers built from registered parts,
a run order over them, a final norm and an LM head.

Nothing here is specific to one architecture: the `ModelConfig` says which
part kinds each layer has and in which order the layers run.  From the mixers'
cache needs it derives the cache groups (layers whose needs are identical share
pages and a block table; layers with a window get pages of their own) and each
run-order entry's binding.

Forward order follows `engine/src/gpu_model.rs:3254-3580` (prefill) and
`:1393-1605` (decode): embed -> layers -> gather wanted rows -> final norm ->
LM head.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..ops import layer_close
from ..config.model_config import ConfigError, ModelConfig
from ..parts import (ARRANGEMENTS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, CacheNeed,
                     LayerBinding, TensorDecl)


@dataclass(frozen=True)
class CacheGroupSpec:
    """Layers whose keys and values share pages: one pool, one block table."""
    need: CacheNeed
    layers: Tuple[int, ...]          # stored-layer indices, in slot order (a layer that runs in
                                     # several copies has a slot for each)


@dataclass(frozen=True)
class TensorRequest:
    key: str                         # "<part path>.<local name>", unique in the model
    checkpoint_name: str
    decl: TensorDecl


class ModelVectors:
    """Tables of the model itself: float32 rows as wide as the model, by name.  A run-order
    entry may add one of their rows to the residual before its layer runs."""

    def __init__(self, tables, width: int):
        self.tables = tuple(tables)
        self.width = width
        self.bound: Dict[str, torch.Tensor] = {}

    def tensors(self):
        return [TensorDecl(name, (rows, self.width), role="vector", init=("normal", 0.0, 0.5))
                for name, rows in self.tables]

    def bind(self, tensors, dtype, device):
        self.bound = {name: tensors[name].contiguous() for name, _ in self.tables}

    def row(self, name: str, index: int) -> torch.Tensor:
        return self.bound[name][index]


class ModelMatrices:
    """Matrices of the model itself, W [width, 2 width] by name: a run-order entry may put the
    residual x and the embedding's output x0 through one of them, x <- W [x; x0].  The part of
    the product that x0 has is the same whenever it is taken, so a step takes it once."""

    def __init__(self, names, width: int):
        self.names = tuple(names)
        self.width = width
        self.halves: Dict[str, Tuple[torch.Tensor, torch.Tensor]] = {}

    def tensors(self):
        return [TensorDecl(name, (self.width, 2 * self.width)) for name in self.names]

    def bind(self, tensors, dtype, device):
        self.dtype = dtype
        for name in self.names:
            w = tensors[name]
            self.halves[name] = (w[:, :self.width].contiguous(), w[:, self.width:].contiguous())
            ops.declare_weights(*self.halves[name])

    def of_embedding(self, ctx, name: str, x: torch.Tensor) -> torch.Tensor:
        """The embedding's share of every later `enter`; `x`: the embedding's output."""
        rows = ctx.scratch("entry.rows", x.shape, self.dtype)
        layer_close.swap_rows(x, rows)
        share = ctx.scratch(f"entry.share.{name}", x.shape, torch.float32)
        ops.linear(rows, self.halves[name][1], share)
        return share

    def enter(self, ctx, name: str, x: torch.Tensor, share: torch.Tensor) -> None:
        rows = ctx.scratch("entry.rows", x.shape, self.dtype)
        layer_close.swap_rows(x, rows, share)
        ops.linear(rows, self.halves[name][0], x, accumulate=True)


class DecoderModel:
    def __init__(self, config: ModelConfig):
        self.config = config
        self.embedding = EMBEDDINGS.build(config.embedding.kind, config.embedding,
                                          config.vocab_size, config.hidden_size)
        self.head = HEADS.build(config.head.kind, config.head, config.vocab_size,
                                config.hidden_size, config.tie_word_embeddings)
        self.final_norm = NORMS.build(config.final_norm.kind, config.final_norm)
        self.vectors = ModelVectors(config.vectors, config.hidden_size)
        self.matrices = ModelMatrices(config.matrices, config.hidden_size)
        self.layers = []
        for spec in config.layers:
            mixer = MIXERS.build(spec.mixer.kind, spec.mixer)
            ffn = FEED_FORWARDS.build(spec.feed_forward.kind, spec.feed_forward)
            norms = {name: NORMS.build(n.kind, n) for name, n in spec.norms}
            self.layers.append(ARRANGEMENTS.build(spec.arrangement, spec, norms, mixer, ffn))
        self.cache_groups, self.bindings, self.state_bytes = self._plan_storage()
        self.dtype: Optional[torch.dtype] = None
        self.device: Optional[torch.device] = None

    # -- storage planning ---------------------------------------------------

    def _plan_storage(self):
        """Cache groups, one binding per run-order entry, state bytes per request."""
        owners: Dict[Tuple[int, int], Tuple[int, int]] = {}   # (stored layer, copy) -> (group, slot)
        groups: List[Tuple[CacheNeed, List[int]]] = []
        # a layer that only ever runs on another layer's cache gets no pages of its own; a
        # layer that runs in several copies gets a slot for each
        runs_on_own = sorted({(e.layer, e.copy) for e in self.config.run_order if e.cache_of is None})
        for li, copy in runs_on_own:
            need = self.layers[li].mixer.cache_need()
            if need is None:
                continue
            for gi, (gneed, members) in enumerate(groups):
                if gneed == need:
                    owners[(li, copy)] = (gi, len(members))
                    members.append(li)
                    break
            else:
                owners[(li, copy)] = (len(groups), 0)
                groups.append((need, [li]))
        bindings: List[LayerBinding] = []
        state_offsets: Dict[Tuple[int, int], int] = {}
        total_state = 0
        # an embedding that remembers something of a request between steps (its last token,
        # say) keeps it at the head of the request's state slot
        nbytes = int(getattr(self.embedding, "state_bytes", lambda: 0)())
        if nbytes:
            self.embedding.state_binding = LayerBinding(state_offset=0, state_bytes=nbytes)
            total_state = (nbytes + 15) // 16 * 16
        written, ran = set(), set()
        for i, entry in enumerate(self.config.run_order):
            layer = self.layers[entry.layer]
            nbytes = int(layer.mixer.state_bytes())
            own = int(getattr(layer, "own_state_bytes", lambda: 0)())
            me = (entry.layer, entry.copy)
            if (nbytes or own) and me not in state_offsets:
                # the mixer's bytes, then the arrangement's own
                state_offsets[me] = total_state
                total_state += (nbytes + 15) // 16 * 16 + (own + 15) // 16 * 16
            group = slot = None
            write = True
            if entry.cache_of is not None:
                src = (entry.cache_of, entry.copy)
                if src not in owners:
                    raise ConfigError(f"run_order[{i}] reads the cache of layer {src[0]}, "
                                      f"whose mixer keeps none")
                if layer.mixer.cache_need() != self.layers[src[0]].mixer.cache_need():
                    raise ConfigError(f"run_order[{i}]: layer {entry.layer} cannot read the "
                                      f"cache of layer {src[0]}: their cache needs differ")
                if src not in written:
                    raise ConfigError(f"run_order[{i}] reads the cache of layer {src[0]} "
                                      f"before that layer has run")
                group, slot = owners[src]
                write = False
            elif me in owners:
                group, slot = owners[me]
                if me in written:
                    raise ConfigError(f"run_order[{i}] runs layer {entry.layer} a second "
                                      f"time and would write its cache twice; name "
                                      f"cache_of to read it instead, or another copy")
                written.add(me)
            if (nbytes or own) and me in ran:
                raise ConfigError(f"run_order[{i}] runs layer {entry.layer} a second time on "
                                  f"the same state; name another copy")
            ran.add(me)
            bindings.append(LayerBinding(group=group, slot=slot or 0, write=write,
                                         state_offset=state_offsets.get(me, 0),
                                         state_bytes=nbytes,
                                         own=LayerBinding(
                                             state_offset=state_offsets[me] + (nbytes + 15) // 16 * 16,
                                             state_bytes=own) if own else None))
        specs = [CacheGroupSpec(need, tuple(members)) for need, members in groups]
        return specs, bindings, total_state

    # -- tensors ------------------------------------------------------------

    def _parts(self):
        """(path, part, layer index or None) for every part that has tensors."""
        yield "embedding", self.embedding, None
        yield "head", self.head, None
        yield "final_norm", self.final_norm, None
        if self.vectors.tables:
            yield "vectors", self.vectors, None
        if self.matrices.names:
            yield "matrices", self.matrices, None
        for li, layer in enumerate(self.layers):
            for name, norm in layer.norms.items():
                yield f"layer.{name}", norm, li
            yield "layer.mixer", layer.mixer, li
            yield "layer.feed_forward", layer.feed_forward, li
            if hasattr(layer, "tensors"):          # an arrangement with weights of its own
                yield "layer.arrangement", layer, li

    def tensor_requests(self) -> List[TensorRequest]:
        names = self.config.tensor_names
        out = []
        for path, part, li in self._parts():
            for decl in part.tensors():
                local = f"{path}.{decl.name}"
                if local not in names:
                    raise ConfigError(f"architecture {self.config.architecture!r} gives no "
                                      f"checkpoint name for {local!r}")
                ckpt = names[local].format(layer=li) if li is not None else names[local]
                key = local if li is None else f"{local}@{li}"
                out.append(TensorRequest(key, ckpt, decl))
        return out

    def bind(self, loaded: Dict[str, Optional[torch.Tensor]], dtype: torch.dtype,
             device: torch.device) -> None:
        self.dtype, self.device = dtype, device
        for path, part, li in self._parts():
            mine = {}
            for decl in part.tensors():
                key = f"{path}.{decl.name}" if li is None else f"{path}.{decl.name}@{li}"
                mine[decl.name] = loaded.get(key)
            part.bind(mine, dtype, device)
        if self.config.tie_word_embeddings:
            self.head.tie(self.embedding.table)
        # a head that scales its logits does so by the gain of the norm its rows come from (a
        # float32 number on the rows before they are rounded)
        scale = float(getattr(self.head, "scale", 1.0))
        if scale != 1.0:
            self.final_norm.scale_gain(scale)

    @property
    def graph_safe(self) -> bool:
        return self._graph_flags()[0]

    @property
    def graph_safe_prompt_steps(self) -> bool:
        return self._graph_flags()[1]

    def _graph_flags(self):
        """(decode steps may be captured, steps with prompt portions may be captured): what
        the parts say about themselves, asked once."""
        flags = self.__dict__.get("_graph_flags_cache")
        if flags is None:
            def prompt_ok(part):
                flag = getattr(part, "graph_safe_prompt_steps", None)
                return getattr(part, "graph_safe", True) if flag is None else flag
            parts = [part for _, part, _ in self._parts()]
            flags = (all(getattr(part, "graph_safe", True) for part in parts),
                     all(prompt_ok(part) for part in parts))
            self._graph_flags_cache = flags
        return flags

    # -- one step -------------------------------------------------------------

    def forward(self, ctx) -> torch.Tensor:
        """Runs the step's tokens; returns fp32 logits [wanted rows, vocab]."""
        x = self.embedding.forward(ctx, ctx.token_ids)
        order = self.config.run_order
        embedded = None
        if any(entry.add_embedding for entry in order):
            embedded = ctx.scratch("embedding.output", x.shape, torch.float32)
            embedded.copy_(x)
        shares = {name: self.matrices.of_embedding(ctx, name, x)
                  for name in self.matrices.names if any(entry.project == name for entry in order)}
        for i, (entry, binding) in enumerate(zip(order, self.bindings)):
            # the norm that reads the rows after this layer, for the layer's last product
            nxt = self.layers[order[i + 1].layer] if i + 1 < len(order) else None
            entry_norm = getattr(nxt, "entry_norm", None)
            # (rows that get a vector added before the next layer are not final when this one ends)
            changed = i + 1 < len(order) and (order[i + 1].add is not None or order[i + 1].add_embedding
                                              or order[i + 1].project is not None)
            ctx.norm_after_layer = entry_norm() if entry_norm is not None and not changed else None
            norms_at_entry = getattr(nxt, "norms_at_entry", None)
            ctx.norms_after_layer = norms_at_entry() if norms_at_entry is not None and not changed else None
            if entry.project is not None:
                self.matrices.enter(ctx, entry.project, x, shares[entry.project])
            vector = self.vectors.row(*entry.add) if entry.add is not None else None
            if entry.add_embedding:
                ops.add_rows(x, embedded, vector)
            elif vector is not None:
                ops.add_vector(x, vector)
            self.layers[entry.layer].forward(ctx, x, binding)
        ctx.norm_after_layer = ctx.norms_after_layer = None
        if ctx.n_logit_rows == 0:
            return ctx.scratch("logits", (0, self.config.vocab_size), torch.float32)
        if x.dim() == 3:
            # a residual of several streams: the model's result is their sum
            from ..ops import streams
            rows = ctx.scratch("head.rows", (ctx.n_logit_rows, self.config.hidden_size),
                               torch.float32)
            streams.sum_rows(x, ctx.logit_rows, rows)
        elif ctx.host.all_single_token and ctx.n_logit_rows == ctx.n_tokens:
            # every request brings one token and wants its logits: the wanted rows are the
            # step's rows in order (a fact of the step's shape, so a captured step replays)
            rows = x
        else:
            rows = ctx.scratch("head.rows", (ctx.n_logit_rows, self.config.hidden_size),
                               torch.float32)
            ops.gather_rows(x, ctx.logit_rows, rows)
        h = self.final_norm.forward(ctx, rows)
        return self.head.forward(ctx, h)
