"""Attention with two softmax maps per head over the same values.

q = h Wq^T + bq [H, 2, D], k = h Wk^T + bk [G, 2, D], v = h Wv^T + bv [G, E]; query head i reads
key/value head i // (H / G).  Map m of head i: softmax over the earlier keys of
(temperature(p) q_im . k_jm) * scale, temperature(p) = 1 + coef * ln(floor((p + 1) / every) + 1);
a_m its mean of the values.  With lambda = exp(sum lq1 lk1) - exp(sum lq2 lk2) + diff, one number
for the layer:  o = a_1 - lambda a_2, divided by its root mean square over E (eps under the root),
times (1 - diff); the heads' results go through Wo, + bo.  No rotation.

Options of the spec: value_dim (default head_dim, the size of ONE map's keys), diff, norm_eps,
bias (default true: `q.b`, `k.b`, `v.b`, `o.b`), q_temp ((coef, every) or None), out_scale (the
mixer's result times this, default 1).  `window` None.

How it runs: a cached key row holds both maps' keys side by side (2D features), a map's query is
zero in the other map's half, so the paged attention of 2H query heads over G key/value heads
gives both maps' results and reads every key and value once for both.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.model_config import MixerSpec
from ..ops import differential as kernels
from ..ops import sink_attention
from .base import MIXERS, CacheNeed, Mixer, TensorDecl


class DifferentialAttention(Mixer):
    def __init__(self, spec: MixerSpec):
        s = self.spec = spec
        self.H, self.G, self.D = s.n_heads, s.n_kv_heads, s.head_dim
        self.E = int(s.option("value_dim", s.head_dim))
        self.eps = float(s.option("norm_eps", 1e-6))
        self.diff = float(s.option("diff", 0.0))
        self.has_bias = bool(s.option("bias", True))
        temp = s.option("q_temp")
        self.coef, self.every = (float(temp[0]), int(temp[1])) if temp is not None else (0.0, 0)
        self.out_scale = float(s.option("out_scale", 1.0))
        if self.H <= 0 or self.G <= 0 or self.H % self.G or self.D <= 0 or self.E <= 0:
            raise ValueError("differential attention: heads must be a multiple of kv_heads; sizes positive")
        if temp is not None and self.every <= 0:
            raise ValueError("differential attention: the temperature's `every` must be positive")
        if s.window is not None or s.position is not None:
            raise ValueError("differential attention has neither a window nor a rotation")

    def tensors(self):
        d, H, G, D, E = self.spec.width, self.H, self.G, self.D, self.E
        sizes = {"q": H * 2 * D, "k": G * 2 * D, "v": G * E}
        out = [TensorDecl(n, (rows, d)) for n, rows in sizes.items()] + [TensorDecl("o", (d, H * E))]
        if self.has_bias:
            out += [TensorDecl(f"{n}.b", (rows,), role="vector", init=("normal", 0.0, 0.1))
                    for n, rows in dict(sizes, o=d).items()]
        out += [TensorDecl(n, (D,), role="vector", init=("normal", 0.0, 0.1)) for n in ("lq1", "lk1", "lq2", "lk2")]
        return out

    def bind(self, tensors, dtype, device):
        rows = [tensors["q"], tensors["k"], tensors["v"]]
        self.w_in = torch.cat(rows, 0).contiguous()
        self.w_out = tensors["o"]
        self.bias = self.out_bias = None
        if self.has_bias:
            self.bias = torch.cat([tensors["q.b"], tensors["k.b"], tensors["v.b"]], 0).contiguous()
            self.out_bias = (tensors["o.b"] * self.out_scale).contiguous()
        pair = lambda a, b: float(torch.exp((tensors[a].double() * tensors[b].double()).sum()))
        self.lam = pair("lq1", "lk1") - pair("lq2", "lk2") + self.diff
        self.dtype = dtype
        ops.declare_weights(self.w_in, self.w_out)

    def cache_need(self):
        two = 2 * self.D
        return CacheNeed(kv_heads=self.G, head_dim=two, value_dim=self.E if self.E != two else None)

    def forward(self, ctx, h, residual, binding):
        t, H, G, D, E = h.shape[0], self.H, self.G, self.D, self.E
        two = 2 * D
        proj = ctx.scratch("differential.proj", (t, self.w_in.shape[0]), self.dtype)
        ops.linear(h, self.w_in, proj)
        cache = ctx.cache(binding.group)
        qx = ctx.scratch("differential.q", (t, 2 * H * two), self.dtype)
        kernels.prepare(proj, self.bias, self.coef, self.every, qx, H, G, D, E, ctx, cache, binding)
        maps = ctx.scratch("differential.maps", (t, 2 * H * E), self.dtype)
        if two == E:
            ops.paged_attention(qx, maps, 2 * H, G, two, self.spec.softmax_scale, None, ctx, cache, binding)
        else:
            sink_attention.attention(qx, None, maps, None, 2 * H, G, two, E, self.spec.softmax_scale, None, 0, 1.0,
                                     ctx, cache, binding)
        act = ctx.scratch("differential.act", (t, H * E), self.dtype)
        kernels.combine(maps, self.lam, self.eps, (1.0 - self.diff) * self.out_scale, act, self.out_bias, residual,
                        H, E)
        ops.linear(act, self.w_out, residual, accumulate=True, closes=ctx)


MIXERS.register("differential_attention", DifferentialAttention)
