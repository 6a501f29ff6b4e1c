"""Block arrangements.  `pre_norm` is the only one the reference runs on the
GPU (`model.py:262-264`, `engine/src/gpu_model.rs:518-520`):
x = x + mixer(norm(x)); x = x + ffn(norm(x)).  `parallel` has one norm that both
sublayers read: with n = norm(x), x = x + mixer(n) + ffn(n).  `parallel_two_norms` gives each of
the two a norm of its own over the same x and may scale their results.  `pre_norm_conv` is `pre_norm`
with a short causal convolution on what each sublayer reads."""
from __future__ import annotations

import torch

from .base import ARRANGEMENTS, Arrangement, TensorDecl


class PreNormBlock(Arrangement):
    norm_names = ("mixer_norm", "feed_forward_norm")

    def __init__(self, spec, norms, mixer, feed_forward):
        # a layer without a feed-forward sublayer (a part with `absent`) has one norm only
        self.has_ffn = not getattr(feed_forward, "absent", False)
        if not self.has_ffn:
            self.norm_names = ("mixer_norm",)
        super().__init__(spec, norms, mixer, feed_forward)

    def forward(self, ctx, x, binding):
        h = self._norm(ctx, self.norms["mixer_norm"], self.mixer, x)
        if not self.has_ffn:
            self._announce(ctx, getattr(ctx, "norm_after_layer", None), x)
            self.mixer.forward(ctx, h, x, binding)
            return
        self._announce(ctx, (self.norms["feed_forward_norm"], self.feed_forward), x)
        self.mixer.forward(ctx, h, x, binding)
        h = self._norm(ctx, self.norms["feed_forward_norm"], self.feed_forward, x)
        self._announce(ctx, getattr(ctx, "norm_after_layer", None), x)
        self.feed_forward.forward(ctx, h, x)

    def entry_norm(self):
        """(norm, its consumer): the first reader of the rows this layer is given."""
        return self.norms["mixer_norm"], self.mixer

    @staticmethod
    def _announce(ctx, ahead, x):
        # the part that runs now writes x last before `ahead`'s norm reads it: its last product
        # may leave that norm's input (StepContext.announce_norm)
        announce = getattr(ctx, "announce_norm", None)
        if announce is None:
            return
        norm, consumer = ahead if ahead is not None else (None, None)
        # (a consumer with `takes_prenormed = False` fuses the norm of a few rows into its first
        # product but has no product that takes rows a product before it left ahead of their norm)
        if (norm is not None and getattr(consumer, "fuses_norm", False)
                and getattr(consumer, "takes_prenormed", True)
                and getattr(norm, "supports_ahead", False)):
            announce(norm, x)
        else:
            announce(None, None)

    @staticmethod
    def _norm(ctx, norm, consumer, x):
        # a consumer that can fuse the norm into its first product (`fuses_norm`)
        # may be handed rows that are not yet normalised, if the norm offers that
        if getattr(consumer, "fuses_norm", False) and getattr(norm, "supports_lazy", False):
            return norm.forward(ctx, x, lazy=True)
        return norm.forward(ctx, x)


class ParallelBlock(Arrangement):
    """One norm, two readers: n = norm(x); x += mixer(n); x += ffn(n).  Both sublayers add
    their results into the fp32 residual, so the layer's sum is a 32-bit sum; the order of
    the two additions is fixed.  A feed-forward part with `absent` leaves the mixer alone."""
    norm_names = ("norm",)

    def __init__(self, spec, norms, mixer, feed_forward):
        self.has_ffn = not getattr(feed_forward, "absent", False)
        super().__init__(spec, norms, mixer, feed_forward)

    def forward(self, ctx, x, binding):
        announce = getattr(ctx, "announce_norm", None)
        if announce is not None:
            announce(None, None)       # the rows' next norm reads them after BOTH sublayers
        n = self.norms["norm"].forward(ctx, x)
        self.mixer.forward(ctx, n, x, binding)
        if self.has_ffn:
            self.feed_forward.forward(ctx, n, x)


class ParallelTwoNormBlock(Arrangement):
    """x += s1 * mixer(mixer_norm(x)) + s2 * ffn(feed_forward_norm(x)), both norms of the same x.
    Option `layer_scale` of the layer: s1 and s2 are the float32 vectors `mixer_scale` and
    `feed_forward_scale` [width] (else ones).  The mixer writes its result beside the residual and
    the feed-forward leaves its sum open; one launch adds both in 32 bits and takes the norms of
    the layer that follows.  The mixer must be able to write instead of add (`can_overwrite`), the
    feed-forward must offer `forward_open`, or be absent."""
    norm_names = ("mixer_norm", "feed_forward_norm")

    def __init__(self, spec, norms, mixer, feed_forward):
        self.has_ffn = not getattr(feed_forward, "absent", False)
        if not self.has_ffn:
            self.norm_names = ("mixer_norm",)
        super().__init__(spec, norms, mixer, feed_forward)
        if not getattr(mixer, "can_overwrite", False):
            raise ValueError("parallel_two_norms: the mixer must be able to write its result")
        if self.has_ffn and not hasattr(feed_forward, "forward_open"):
            raise ValueError("parallel_two_norms: the feed-forward must leave its sum open")
        self.width = spec.mixer.width
        self.scaled = bool(spec.option("layer_scale", False))
        self.scales = {}

    def tensors(self):
        if not self.scaled:
            return []
        return [TensorDecl(f"{name}_scale", (self.width,), role="vector", init=("normal", 0.8, 0.2))
                for name in (("mixer", "feed_forward") if self.has_ffn else ("mixer",))]

    def bind(self, tensors, dtype, device):
        self.scales = {name: t.contiguous() for name, t in tensors.items() if t is not None}

    def norms_at_entry(self):
        """The norms that read the rows this layer is given, in the order of `norm_names`."""
        return tuple(self.norms[name] for name in self.norm_names)

    def forward(self, ctx, x, binding):
        from ..ops import layer_close
        announce = getattr(ctx, "announce_norm", None)
        if announce is not None:
            announce(None, None)
        mine = self.norms_at_entry()
        if ctx.take_closed(x, mine):
            h = self._rows(ctx, x, mine)
        else:
            h = self._rows(ctx, x, mine)
            layer_close.close(x, None, None, None, None, self._norm_args(mine, h))
        mixed = ctx.scratch("layer.mixed", x.shape, torch.float32)
        self.mixer.forward(ctx, h[0], mixed, binding, accumulate=False)
        left = self.feed_forward.forward_open(ctx, h[1]) if self.has_ffn else None
        after = getattr(ctx, "norms_after_layer", None) or ()
        layer_close.close(x, mixed, self.scales.get("mixer_scale"), left, self.scales.get("feed_forward_scale"),
                          self._norm_args(after, self._rows(ctx, x, after)))
        if after:
            ctx.offer_closed(x, after)

    @staticmethod
    def _rows(ctx, x, norms):
        return [ctx.scratch(f"layer.normed{i}", x.shape, norm.dtype) for i, norm in enumerate(norms)]

    @staticmethod
    def _norm_args(norms, rows):
        return [(norm.gain, norm.spec.eps, out) for norm, out in zip(norms, rows)]


class PreNormConvBlock(PreNormBlock):
    """x += mixer(c1(norm(x))); x += ffn(c2(norm(x))), c(h)_t = h_t + sum_j w_j h_(t - taps + 1 + j)
    along a request's tokens, channel by channel (zeros before its start).  Norm, convolution and
    sum are one launch, in 32 bits.  Option `taps` of the layer; tensors `mixer_conv` and
    `feed_forward_conv` [width, taps] (the last column meets the current token).  The last
    taps - 1 rows h of both sublayers are state of the layer's run."""

    def __init__(self, spec, norms, mixer, feed_forward):
        super().__init__(spec, norms, mixer, feed_forward)
        self.taps = int(spec.option("taps", 4))
        if not 1 <= self.taps <= 64:
            raise ValueError(f"pre_norm_conv: 1 to 64 taps, got {self.taps}")
        self.width = spec.mixer.width
        self.tail_bytes = (4 * (self.taps - 1) * self.width + 15) // 16 * 16
        self.conv = {}
        self.dtype = None

    @property
    def sublayers(self):
        return ("mixer", "feed_forward") if self.has_ffn else ("mixer",)

    def tensors(self):
        return [TensorDecl(f"{s}_conv", (self.width, self.taps), role="vector", init=("uniform", -0.5, 0.5))
                for s in self.sublayers]

    def bind(self, tensors, dtype, device):
        self.dtype = dtype
        # tap by tap, so that neighbouring columns lie side by side
        self.conv = {s: tensors[f"{s}_conv"].t().contiguous() for s in self.sublayers}

    def own_state_bytes(self) -> int:
        return self.tail_bytes * len(self.sublayers)

    def entry_norm(self):
        return None          # the norm's rows go through the convolution: no product takes them as they are

    def forward(self, ctx, x, binding):
        announce = getattr(ctx, "announce_norm", None)
        if announce is not None:
            announce(None, None)
        self.mixer.forward(ctx, self._read(ctx, x, binding, "mixer", 0), x, binding)
        if not self.has_ffn:
            return
        h = self._read(ctx, x, binding, "feed_forward", self.tail_bytes)
        self._announce(ctx, getattr(ctx, "norm_after_layer", None), x)
        self.feed_forward.forward(ctx, h, x)

    def _read(self, ctx, x, binding, sublayer, tail_off):
        from ..ops import input_conv
        norm = self.norms[f"{sublayer}_norm"]
        out = ctx.scratch("norm.out", x.shape, self.dtype)
        state = ctx.state(binding.own) if binding.own is not None else None
        input_conv.norm_conv(x, norm.gain, norm.spec.eps, self.conv[sublayer], ctx, state, tail_off, out)
        return out


ARRANGEMENTS.register("pre_norm", PreNormBlock)
ARRANGEMENTS.register("pre_norm_conv", PreNormConvBlock)
ARRANGEMENTS.register("parallel", ParallelBlock)
ARRANGEMENTS.register("parallel_two_norms", ParallelTwoNormBlock)
