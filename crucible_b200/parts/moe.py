"""Feed-forwards of this family: a dense one with a chosen activation, and a mixture of
experts.

`dense_act`: x += act(h Wup^T) Wdown^T; the activation is an option of the spec (relu2:
the square of ReLU; gelu_tanh; silu; tanh).

`glu_capped`: x += pair(h Wg^T, h Wu^T) Wdown^T with the capped gated pair: g' = min(g, limit),
u' = clamp(u, -limit, limit), pair = g' * sigmoid(alpha * g') * (u' + offset); `limit`, `alpha`
(default 1.702) and `offset` (default 1) are options of the spec.

`moe`: `experts` gated feed-forwards Wd_e (silu(Wg_e h) * (Wu_e h)) without biases, of
which a token uses the `top` with the largest router logits z = h Wr^T (float32; the lower
index on ties), weighted by the softmax over those `top` logits alone; an optional shared
expert of the same form runs for every token and is added.  Options: `router_bias` (the
logits are h Wr^T + b, tensor `router.b`), `pair` = (limit, alpha, offset): the experts use
the capped gated pair instead of silu(g) * u; `groups` = (count, keep): the experts form `count`
equal groups of neighbours, a group's score is its best logit, and only the experts of the `keep`
best groups can be chosen; `shared_gate` (tensor `shared.sg` [1, width]): the shared expert's result
is multiplied by sigmoid(h Wsg^T), one number a token; `out_scale`: everything times this number;
`score` = "sigmoid": with s = sigmoid(z) the experts with the largest s + `correction` (a float32
vector) are chosen and weighted by s as it is; `group_score` = "two_best": a group's score is the sum
of its two best scores (default "best").  `forward_open` leaves the sum to the caller (an arrangement
that scales it and adds a mixer's result in the same pass), the shared expert included.
(The softmax over the chosen logits alone is the chosen experts' softmax over all experts divided
by their sum.)
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.model_config import FeedForwardSpec
from ..ops import moe as kernels
from ..ops.layer_close import OpenSum
from .base import FEED_FORWARDS, FeedForward, TensorDecl
from .swiglu import SwiGLU


class ActivatedFeedForward(FeedForward):
    fuses_norm = True          # h goes into one product: few rows are normalised on their way in
    takes_prenormed = False

    def __init__(self, spec: FeedForwardSpec):
        self.spec = spec
        self.kind = str(spec.option("activation", "relu2"))
        if self.kind not in ops.ACTIVATIONS:
            raise ValueError(f"dense_act: unknown activation {self.kind!r}; known: {sorted(ops.ACTIVATIONS)}")
        self.up = self.down = None

    def tensors(self):
        d, f = self.spec.width, self.spec.intermediate
        return [TensorDecl("up", (f, d)), TensorDecl("down", (d, f))]

    def bind(self, tensors, dtype, device):
        self.up, self.down = tensors["up"], tensors["down"]
        ops.declare_weights(self.up, self.down)
        self.dtype = dtype

    def forward(self, ctx, h, residual):
        z = ctx.scratch("ffn.z", (h.shape[0], self.spec.intermediate), self.dtype)
        ops.linear_act(h, self.up, z, self.kind)
        ops.linear(z, self.down, residual, accumulate=True, closes=ctx)


class CappedGLU(FeedForward):
    fuses_norm = True
    takes_prenormed = False

    def __init__(self, spec: FeedForwardSpec):
        self.spec = spec
        self.limit = float(spec.option("limit", 0.0))
        self.alpha = float(spec.option("alpha", 1.702))
        self.offset = float(spec.option("offset", 1.0))
        if not self.limit > 0:
            raise ValueError("glu_capped: the limit must be positive")
        self.gate_up = self.down = None

    def tensors(self):
        d, f = self.spec.width, self.spec.intermediate
        return [TensorDecl("gate", (f, d)), TensorDecl("up", (f, d)), TensorDecl("down", (d, f))]

    def bind(self, tensors, dtype, device):
        self.gate_up = torch.cat([tensors["gate"], tensors["up"]], dim=0).contiguous()
        self.down = tensors["down"]
        ops.declare_weights(self.gate_up, self.down)
        self.dtype = dtype

    def forward(self, ctx, h, residual):
        t, f = h.shape[0], self.spec.intermediate
        act = ctx.scratch("ffn.act", (t, f), self.dtype)
        ops.linear_swiglu(h, self.gate_up, act, ctx, pair=(self.limit, self.alpha, self.offset))
        ops.linear(act, self.down, residual, accumulate=True, closes=ctx)


class MixtureOfExperts(FeedForward):
    # Nothing of a step's routing comes to the host: the launches depend on the step's shape
    # alone, so prompt steps are captured as graphs like decode steps.
    SMALL_MAX_PAIRS = 256        # up to this many pairs the experts' weight rows are read by a warp each
    SORTED_MIN_PAIRS = 16        # from this many (token, expert) pairs on, the experts run as two
                                 # grouped products over their rows side by side (8 experts of 4096 x
                                 # 2048, two a token: 8 rows 133 us against 152 with a warp per weight
                                 # row, 16 rows 121 against 259, 64 rows 129 against 784)
    MAX_EXPERTS = 256
    RIDE_GROUPED_ROWS = 32       # the same where the experts run as grouped products (a decode step of 16 rows,
                                 # 4 layers of width 1024: 0.379 -> 0.347 ms; at 64 rows of width 2048 no gain)
    RIDE_MAX_ROWS = 2            # up to this many bfloat16 rows a joining shared expert rides with the routed ones

    def __init__(self, spec: FeedForwardSpec):
        self.spec = spec
        self.n = int(spec.option("experts", 0))
        self.top = int(spec.option("top", 0))
        self.ff = int(spec.intermediate)
        shared = spec.option("shared_intermediate")
        self.has_bias = bool(spec.option("router_bias", False))
        self.shared_gate = bool(spec.option("shared_gate", False))
        self.out_scale = float(spec.option("out_scale", 1.0))
        self.score = str(spec.option("score", "softmax"))
        self.group_score = str(spec.option("group_score", "best"))
        if self.score not in ("softmax", "sigmoid") or self.group_score not in ("best", "two_best"):
            raise ValueError(f"moe: score is 'softmax' or 'sigmoid', group_score 'best' or 'two_best', got "
                             f"{self.score!r} and {self.group_score!r}")
        groups = spec.option("groups")
        self.groups = (int(groups[0]), int(groups[1])) if groups is not None else None
        pair = spec.option("pair")
        self.pair = tuple(float(v) for v in pair) if pair is not None else None
        if self.pair is not None and (len(self.pair) != 3 or not self.pair[0] > 0):
            raise ValueError("moe: pair is (limit > 0, alpha, offset)")
        if self.n <= 0 or not 0 < self.top <= self.n or self.ff <= 0:
            raise ValueError("moe: experts, top (at most experts) and the experts' ff must be positive")
        if self.n > self.MAX_EXPERTS or self.top > 32:
            raise ValueError("moe: up to 256 experts, of which a token uses up to 32")
        if self.groups is not None:
            count, keep = self.groups
            if count <= 0 or self.n % count or not 0 < keep <= count or self.top > keep * (self.n // count):
                raise ValueError("moe: groups = (count, keep): count divides the experts, keep is at most "
                                 "count, and the kept groups hold at least `top` experts")
        if shared and self.shared_gate and self.pair is not None:
            raise ValueError("moe: a gated shared expert has no capped pair")
        if shared and not self.shared_gate and self.out_scale != 1.0:
            raise ValueError("moe: a shared expert without a gate takes no out_scale")
        self.shared_ff = int(shared) if shared else 0
        self.shared_gate = self.shared_gate and self.shared_ff > 0
        # a shared expert that joins the experts' sum: one with a gate, or one of a caller that
        # takes the sum open
        self.joins = self.shared_ff > 0 and (self.shared_gate or bool(spec.option("open_sum", False)))
        if self.joins and self.pair is not None:
            raise ValueError("moe: a shared expert that joins the experts' sum has no capped pair")
        self.shared = (SwiGLU(FeedForwardSpec(kind="swiglu", width=spec.width, intermediate=self.shared_ff))
                       if shared and not self.joins else None)
        # A joining shared expert as slices of an expert's size (the last one padded with zeros) that
        # every token chooses: a few rows then take no launches of their own for it.
        self.slices = -(-self.shared_ff // self.ff) if self.joins else 0
        if self.slices > 32 or self.n + self.slices > self.MAX_EXPERTS:
            self.slices = 0

    def tensors(self):
        d, f = self.spec.width, self.ff
        out = [TensorDecl("router", (self.n, d))]
        if self.has_bias:
            out.append(TensorDecl("router.b", (self.n,), role="vector", init=("normal", 0.0, 0.5)))
        if self.score == "sigmoid":
            out.append(TensorDecl("correction", (self.n,), role="vector", init=("normal", 0.0, 0.5)))
        for e in range(self.n):
            out += [TensorDecl(f"e{e}.gate", (f, d)), TensorDecl(f"e{e}.up", (f, d)),
                    TensorDecl(f"e{e}.down", (d, f))]
        if self.shared is not None:
            out += [TensorDecl(f"shared.{t.name}", t.shape, t.role) for t in self.shared.tensors()]
        elif self.joins:
            fs = self.shared_ff
            out += [TensorDecl("shared.gate", (fs, d)), TensorDecl("shared.up", (fs, d)),
                    TensorDecl("shared.down", (d, fs))]
            if self.shared_gate:
                out.append(TensorDecl("shared.sg", (1, d)))
        return out

    def bind(self, tensors, dtype, device):
        self.dtype = dtype
        d, f = self.spec.width, self.ff
        # the router's rows and, behind them, the row of the shared expert's gate: one product
        self.router = (torch.cat([tensors["router"], tensors["shared.sg"]], 0).contiguous()
                       if self.shared_gate else tensors["router"])
        self.router_bias = tensors.get("router.b") if self.has_bias else None
        self.correction = tensors.get("correction") if self.score == "sigmoid" else None
        gate_up = [torch.cat([tensors[f"e{e}.gate"], tensors[f"e{e}.up"]], 0) for e in range(self.n)]
        down = [tensors[f"e{e}.down"] for e in range(self.n)]
        for s in range(self.slices):
            lo, hi = s * f, min((s + 1) * f, self.shared_ff)
            gu, dn = torch.zeros((2 * f, d), dtype=dtype, device=device), torch.zeros((d, f), dtype=dtype, device=device)
            gu[:hi - lo], gu[f:f + hi - lo] = tensors["shared.gate"][lo:hi], tensors["shared.up"][lo:hi]
            dn[:, :hi - lo] = tensors["shared.down"][:, lo:hi]
            gate_up.append(gu)
            down.append(dn)
        self.gate_up = torch.stack(gate_up, 0).contiguous()          # [E + slices, 2F, d]
        self.down = torch.stack(down, 0).contiguous()                # [E + slices, d, F]
        ops.declare_weights(self.router, self.gate_up, self.down)
        # the shared expert as dense products, for steps of many rows
        self.dense = []
        if self.joins:
            if self.slices:
                self.dense = [(self.gate_up[self.n + s], self.down[self.n + s]) for s in range(self.slices)]
            else:
                self.dense = [(torch.cat([tensors["shared.gate"], tensors["shared.up"]], 0).contiguous(),
                               tensors["shared.down"])]
                ops.declare_weights(*self.dense[0])
        self.count = torch.zeros(self.n + self.slices, dtype=torch.int32, device=device)     # zero between steps
        if self.shared is not None:
            self.shared.bind({k[len("shared."):]: v for k, v in tensors.items() if k.startswith("shared.")},
                             dtype, device)

    def forward(self, ctx, h, residual):
        o = self.forward_open(ctx, h)
        kernels.combine(o.rows, o.top, residual, by_plan=o.by_plan, shared=o.shared, gate=o.gate)
        if self.shared is not None:
            self.shared.forward(ctx, h, residual)

    def forward_open(self, ctx, h) -> OpenSum:
        """The experts' rows and what the shared expert adds if it joins their sum, not yet summed."""
        t, d, f = h.shape[0], self.spec.width, self.ff
        logits = ctx.scratch("moe.logits", (t, self.router.shape[0]), torch.float32)
        ops.linear(h, self.router, logits)
        # more than a few rows: the experts' rows side by side and two grouped products on the tensor
        # cores, by the plan on the device (tiles of 128 rows); a joining shared expert then
        # runs as dense products of its own
        grouped = (self.dtype == torch.bfloat16 and d % 8 == 0 and f % 8 == 0
                   and t * self.top >= self.SORTED_MIN_PAIRS)
        most = (self.RIDE_GROUPED_ROWS if grouped else self.RIDE_MAX_ROWS) if self.dtype == torch.bfloat16 else t
        riding = self.slices if t <= most else 0
        apart = self.joins and not riding
        n, top = self.n + riding, self.top + riding              # experts of the plan, pairs of a token
        tile_rows = kernels.GROUPED_TILE_ROWS if grouped else 0
        tiles = kernels.max_tiles(t, top, n, tile_rows)
        idx = ctx.scratch("moe.idx", (t * top,), torch.int32)
        place = ctx.scratch("moe.place", (t * top,), torch.int32)
        order = ctx.scratch("moe.order", (t * top,), torch.int32)
        weight = ctx.scratch("moe.weight", (t * top,), torch.float32)
        plan = ctx.scratch("moe.plan", (kernels.plan_ints(n, tiles),), torch.int32)
        gate = ctx.scratch("moe.shared_gate", (t,), torch.float32) if apart and self.shared_gate else None
        kernels.route(logits, self.top, idx, weight, place, self.count, plan, tiles, order, bias=self.router_bias,
                      rows=tile_rows, n_experts=self.n, groups=self.groups, n_shared=riding,
                      gate_col=self.n if self.shared_gate else -1, scale=self.out_scale, gate_out=gate,
                      sigmoid=self.score == "sigmoid", correction=self.correction,
                      group_best_two=self.group_score == "two_best")
        act = ctx.scratch("moe.act", (t * top, f), self.dtype)
        by_plan = None
        if grouped:
            rows = ctx.scratch("moe.rows", (t * top, d), self.dtype)
            kernels.gather(h, order, top, rows)
            pair_out = ctx.scratch("moe.down", (t * top, d), torch.float32)
            if not (kernels.grouped_linear(rows, self.gate_up, act, plan, n, tiles, True, pair=self.pair)
                    and kernels.grouped_linear(act, self.down, pair_out, plan, n, tiles, False)):
                raise RuntimeError("moe: the grouped product refused sizes its rule allows")
            by_plan = (plan, idx, place, weight)
        else:
            pair_out = ctx.scratch("moe.pair_out", (t * top, d), torch.float32)
            # few rows (decoded tokens): the weights are what moves; a warp per weight row
            small = self.dtype == torch.bfloat16 and t * top <= self.SMALL_MAX_PAIRS
            if not (small and kernels.expert_rows_small(True, h, self.gate_up, f, plan, n, tiles, order, top, weight,
                                                        act, pair=self.pair)):
                kernels.expert_tiles(True, h, self.gate_up, f, plan, n, tiles, order, top, weight, act,
                                     pair=self.pair)
            if not (small and kernels.expert_rows_small(False, act, self.down, d, plan, n, tiles, order, top, weight,
                                                        pair_out)):
                kernels.expert_tiles(False, act, self.down, d, plan, n, tiles, order, top, weight, pair_out)
        shared_out = None
        if apart:
            shared_out = ctx.scratch("moe.shared_out", (t, d), torch.float32)
            for i, (gate_up, down) in enumerate(self.dense):
                shared_act = ctx.scratch("moe.shared_act", (t, down.shape[1]), self.dtype)
                ops.linear_swiglu(h, gate_up, shared_act, ctx)
                ops.linear(shared_act, down, shared_out, accumulate=i > 0)
        return OpenSum(rows=pair_out, top=top, by_plan=by_plan, shared=shared_out, gate=gate)


FEED_FORWARDS.register("dense_act", ActivatedFeedForward)
FEED_FORWARDS.register("glu_capped", CappedGLU)
FEED_FORWARDS.register("moe", MixtureOfExperts)
