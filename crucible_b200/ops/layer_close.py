"""Wrappers of `csrc/layer_close.cu`: the sum that ends a layer with the norms of what follows, and
the rows of a repeated run's entry."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import torch

from . import KernelError, _c_float, _c_int, _check, _code, _contig, _need_cuda, _ptr, _stream, build


@dataclass
class OpenSum:
    """A feed-forward's result before its sum: the experts' rows (float32; `top` of them a token, by
    pair and weighted, or with `by_plan` = (plan, idx, place, weight) in the sorted order) and rows
    by token (`shared`) that join with `gate` (float32 [tokens]; None: as they are)."""
    rows: Optional[torch.Tensor] = None
    top: int = 0
    by_plan: Optional[tuple] = None
    shared: Optional[torch.Tensor] = None
    gate: Optional[torch.Tensor] = None


def close(x: torch.Tensor, mixer: Optional[torch.Tensor], s1: Optional[torch.Tensor], open_sum: Optional[OpenSum],
          s2: Optional[torch.Tensor], norms: Sequence[Tuple[torch.Tensor, float, torch.Tensor]] = ()) -> None:
    """x += s1 * mixer + s2 * (the open sum); then each of `norms` = (gain, eps, out), at most two:
    out = rmsnorm(x) * gain.  Everything but x may be absent."""
    o = open_sum if open_sum is not None else OpenSum()
    plan, idx, place, weight = o.by_plan if o.by_plan is not None else (None,) * 4
    _need_cuda(x, mixer, s1, s2, o.rows, plan, idx, place, weight, o.shared, o.gate,
               *(t for n in norms for t in (n[0], n[2])))
    width = x.shape[1]
    for t, what in ((x, "rows"), (mixer, "mixer"), (o.rows, "experts' rows"), (o.shared, "shared rows")):
        if t is None:
            continue
        if t.dtype != torch.float32 or t.dim() != 2 or t.shape[1] != width:
            raise KernelError(f"layer close: the {what} are float32 [*, {width}]")
        _contig(t, "layer close " + what)
    if any(t is not None and t.shape != x.shape for t in (mixer, o.shared)) \
            or (o.rows is not None and o.rows.shape[0] < x.shape[0] * o.top):
        raise KernelError("layer close: results of another number of tokens")
    for v in (s1, s2) + tuple(n[0] for n in norms):
        if v is not None and (v.dtype != torch.float32 or v.numel() != width or not v.is_contiguous()):
            raise KernelError("layer close: scales and gains are float32 vectors over the width")
    outs = [n[2] for n in norms]
    if len(norms) > 2 or any(t.shape != x.shape or not t.is_contiguous() or t.dtype != outs[0].dtype for t in outs):
        raise KernelError("layer close: at most two norms, each into rows of one dtype")
    padded = list(norms) + [(None, 0.0, None)] * (2 - len(norms))
    lib = build.load("layer_close")
    _check(lib.cb_layer_close(
        _ptr(x), _ptr(mixer), _ptr(s1), _ptr(s2), _ptr(o.rows), _c_int(o.top), _ptr(plan), _ptr(idx), _ptr(place),
        _ptr(weight), _ptr(o.shared), _ptr(o.gate), _c_int(len(norms)),
        *(a for g, eps, out in padded for a in (_ptr(g), _c_float(eps), _ptr(out))),
        _c_int(_code(outs[0].dtype) if outs else 0), _c_int(x.shape[0]), _c_int(width), _stream()), "layer close")


def swap_rows(x: torch.Tensor, rows_out: torch.Tensor, next_rows: Optional[torch.Tensor] = None) -> None:
    """rows_out = x in the dtype of `rows_out`; then x = next_rows if given."""
    _need_cuda(x, rows_out, next_rows)
    if x.dtype != torch.float32 or x.dim() != 2 or rows_out.shape != x.shape or \
            (next_rows is not None and (next_rows.dtype != torch.float32 or next_rows.shape != x.shape)):
        raise KernelError("swap_rows takes float32 rows and writes as many")
    for t in (x, rows_out, next_rows):
        if t is not None:
            _contig(t, "swap_rows rows")
    lib = build.load("layer_close")
    _check(lib.cb_swap_rows(_ptr(x), _ptr(rows_out), _c_int(_code(rows_out.dtype)), _ptr(next_rows),
                            _c_int(x.shape[0]), _c_int(x.shape[1]), _stream()), "swap_rows")
