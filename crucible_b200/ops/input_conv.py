"""Wrapper of `csrc/input_conv.cu`: RMS norm and a short causal convolution over time on what
it leaves, added to it, whose last inputs are part of a request's state."""
from __future__ import annotations

import torch

from . import KernelError, _c_float, _c_int, _check, _code, _contig, _need_cuda, _ptr, _stream, build
from .recurrent import _c_long, _state_args


def norm_conv(x, gain, eps: float, taps_weight, ctx, state, tail_off: int, out) -> None:
    """out[t] = h[t] + sum_j taps_weight[j] * h[t - taps + 1 + j], h = rmsnorm(x) * gain, along each
    request's tokens; `taps_weight` float32 [taps, width], the last row meets the current token.
    `state`: uint8 [slots, bytes] with float32 [taps - 1, width] at `tail_off`: the request's last
    rows h, read for a portion's first tokens and rewritten (None with one tap)."""
    _need_cuda(x, gain, taps_weight, state, out)
    if (x.dtype != torch.float32 or gain.dtype != torch.float32 or taps_weight.dtype != torch.float32
            or taps_weight.shape[1:] != x.shape[1:] or gain.shape[0] != x.shape[1] or out.shape != x.shape):
        raise KernelError("norm_conv takes float32 rows, gains and taps of one width")
    for t, what in ((x, "rows"), (gain, "gain"), (taps_weight, "taps"), (out, "output")):
        _contig(t, "norm_conv " + what)
    taps = taps_weight.shape[0]
    sp, stride = _ptr(None), _c_long(0)
    if taps > 1:
        sp, stride = _state_args(state)
        if state.shape[1] < tail_off + 4 * (taps - 1) * x.shape[1]:
            raise KernelError("norm_conv: the state is too small for the convolution's inputs")
    lib = build.load("input_conv")
    _check(lib.cb_norm_conv(
        _ptr(x), _ptr(gain), _c_float(eps), _ptr(taps_weight), _c_int(taps), _ptr(ctx.req_row_start),
        _ptr(ctx.req_state_slot), sp, stride, _c_long(tail_off), _ptr(out), _c_int(_code(out.dtype)),
        _c_int(ctx.n_requests), _c_int(ctx.host.max_new_tokens), _c_int(x.shape[1]), _stream()), "norm_conv")
