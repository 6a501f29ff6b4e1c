"""Wrappers of `csrc/differential.cu`: what surrounds the attention with two softmax maps per
head (biases, the queries' temperature, the two maps' places in one key row; the maps' difference
and its norm)."""
from __future__ import annotations

from typing import Optional

import torch

from . import KernelError, _c_float, _c_int, _check, _code, _need_cuda, _ptr, _stream, build


def prepare(proj, bias: Optional[torch.Tensor], coef: float, every: int, qx, n_heads: int, n_kv_heads: int,
            dim: int, value_dim: int, ctx, cache, binding) -> None:
    """Rows of `proj` are [q: H*2*D | k: G*2*D | v: G*E | ...], `bias` float32 over those columns or
    None.  qx [T, 2H * 2D] = (q + bias) * (1 + coef * ln(floor((p + 1) / every) + 1)) (`every` 0:
    times 1), head h's map m in features m*D .. m*D + D - 1 of head 2h + m, zeros elsewhere; k and v
    with their biases go to the token's place in the pages (keys of 2D features)."""
    _need_cuda(proj, bias, qx)
    two = 2 * dim
    cols = n_heads * two + n_kv_heads * (two + value_dim)
    if proj.stride(1) != 1 or qx.stride(1) != 1 or qx.dtype != proj.dtype or proj.shape[1] < cols \
            or qx.shape != (proj.shape[0], 2 * n_heads * two):
        raise KernelError("differential prepare: rows [q | k | v] and spread queries of one dtype")
    if bias is not None and (bias.dtype != torch.float32 or bias.numel() != cols or not bias.is_contiguous()):
        raise KernelError("differential prepare: one float32 bias for every column of q, k and v")
    k_cache, v_cache = cache.keys(binding.slot), cache.values(binding.slot)
    if k_cache.dtype != proj.dtype or k_cache.shape[-1] != two or v_cache.shape[-1] != value_dim:
        raise KernelError("differential prepare: the pages' sizes or dtype differ from the heads'")
    table = ctx.block_table(binding.group)
    lib = build.load("differential")
    _check(lib.cb_differential_prepare(
        _ptr(proj), _c_int(proj.stride(0)), _c_int(_code(proj.dtype)), _ptr(bias), _c_float(coef), _c_int(every),
        _ptr(ctx.positions), _ptr(ctx.row_request), _ptr(table), _c_int(table.shape[1]), _ptr(qx),
        _c_int(qx.stride(0)), _ptr(k_cache), _ptr(v_cache), _c_int(proj.shape[0]), _c_int(n_heads),
        _c_int(n_kv_heads), _c_int(dim), _c_int(value_dim), _c_int(cache.page_tokens),
        _c_int(1 if binding.write else 0), _stream()), "differential_prepare")


def combine(a, lam: float, eps: float, scale: float, out, out_bias: Optional[torch.Tensor], residual,
            n_heads: int, value_dim: int) -> None:
    """Per head o = a[2h] - lam * a[2h + 1], out = o / sqrt(mean(o^2) + eps) * scale; `out_bias`
    (float32 [width] or None) is added to the float32 residual rows."""
    _need_cuda(a, out, out_bias, residual)
    if (a.dtype != out.dtype or a.stride(1) != 1 or out.stride(1) != 1 or a.shape[1] != 2 * n_heads * value_dim
            or out.shape != (a.shape[0], n_heads * value_dim)):
        raise KernelError("differential combine: rows of 2H and of H heads' values of one dtype")
    if out_bias is not None and (residual.dtype != torch.float32 or not residual.is_contiguous()
                                 or out_bias.dtype != torch.float32 or out_bias.numel() != residual.shape[1]
                                 or residual.shape[0] != a.shape[0]):
        raise KernelError("differential combine: a float32 bias as wide as the float32 residual rows")
    lib = build.load("differential")
    _check(lib.cb_differential_combine(
        _ptr(a), _c_int(a.stride(0)), _c_int(_code(a.dtype)), _c_float(lam), _c_float(eps), _c_float(scale),
        _ptr(out), _c_int(out.stride(0)), _ptr(out_bias), _ptr(residual),
        _c_int(residual.shape[1] if residual is not None else 0), _c_int(a.shape[0]), _c_int(n_heads),
        _c_int(value_dim), _stream()), "differential_combine")
