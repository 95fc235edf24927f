"""Hyper-connections: several parallel residual streams around pre-normed sublayers — csrc/norm/hyper_norm.cu.

The streams of a token are fp32 ``[S, W]``.  A sublayer reads ``u = sum_s a_s x_s`` through a layer norm and its output y joins
all streams at once: ``x_t <- sum_s M[s, t] x_s + b_t y``.  ``hyper_embed`` starts the streams as copies of the scaled embedding;
``hyper_step`` applies one sublayer's update and forms the next sublayer's input in the same pass over the streams;
``hyper_output`` forms the normed sum of the streams for selected rows.  CPU tensors run the PyTorch restatements below (CPU
tests); on a GPU a missing kernel raises.

Reference: none — the reference has no model code (reference llmctl/runtime/engine.py:119-140)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import native
from .elementwise import _is32, _layernorm

c_void_p, c_int, c_ll, c_float = native.c_void_p, native.c_int, native.c_ll, native.c_float
native.register_signature("llmctl_hyper_step", [c_void_p, c_int, c_void_p, c_int, c_ll, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
                                                 c_int, c_void_p, c_void_p, c_int, c_int, c_float, c_void_p])
native.register_signature("llmctl_hyper_embed", [c_void_p, c_void_p, c_int, c_float, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
                                                  c_void_p, c_int, c_int, c_float, c_void_p])
MAX_STREAMS = 16


@dataclass
class StreamWeights:
    """One sublayer's stream weights, fp32: ``a`` [S] (what it reads), ``b`` [S] (where its output goes), ``mix`` [S, S] indexed
    [from, to]."""
    a: torch.Tensor
    b: torch.Tensor
    mix: torch.Tensor


@dataclass
class NextNorm:
    """What the sublayer that follows reads: stream weights ``a`` [S] (None: the plain sum) and layer norm ``w``, ``bias`` [W], fp32;
    ``want_fp32``: also unrounded (a router)."""
    a: Optional[torch.Tensor]
    w: torch.Tensor
    bias: torch.Tensor
    want_fp32: bool = False


Normed = Tuple[Optional[torch.Tensor], Optional[torch.Tensor]]


def _outputs(n: int, W: int, act_dtype: torch.dtype, nxt: Optional[NextNorm], device) -> Normed:
    if nxt is None:
        return None, None
    out = torch.empty(n, W, dtype=act_dtype, device=device)
    return out, (torch.empty(n, W, dtype=torch.float32, device=device) if nxt.want_fp32 and act_dtype != torch.float32 else None)


def _pair(out: Optional[torch.Tensor], out32: Optional[torch.Tensor], nxt: Optional[NextNorm]) -> Normed:
    return out, (out if out32 is None else out32) if nxt is not None and nxt.want_fp32 else None


def _norm_cpu(u: torch.Tensor, nxt: NextNorm, eps: float, act_dtype: torch.dtype) -> Normed:
    h32 = _layernorm(u, nxt.w, nxt.bias, eps)
    h = h32.to(act_dtype)
    return h, h32 if nxt.want_fp32 else None


def hyper_embed(tokens: torch.Tensor, table: torch.Tensor, scale: float, S: int, nxt: Optional[NextNorm], eps: float) -> Tuple[torch.Tensor, Normed]:
    """Streams fp32 [T, S, W], every one ``scale * table[tokens]``, and the first sublayer's input (in the table's type, fp32 or
    None)."""
    T, W = tokens.numel(), table.shape[1]
    if table.is_cuda:
        x = torch.empty(T, S, W, dtype=torch.float32, device=table.device)
        out, out32 = _outputs(T, W, table.dtype, nxt, table.device)
        native.call("llmctl_hyper_embed", tokens.data_ptr(), table.data_ptr(), _is32(table), float(scale), x.data_ptr(), S,
                    native.ptr(nxt.a) if nxt else None, native.ptr(nxt.w) if nxt else None, native.ptr(nxt.bias) if nxt else None,
                    native.ptr(out), native.ptr(out32), T, W, float(eps), native.stream_ptr())
        return x, _pair(out, out32, nxt)
    v = table[tokens.reshape(-1)].float() * scale
    x = v[:, None, :].repeat(1, S, 1)
    if nxt is None:
        return x, (None, None)
    return x, _norm_cpu(v * (nxt.a.sum() if nxt.a is not None else float(S)), nxt, eps, table.dtype)


def _check(x: torch.Tensor, y: Optional[torch.Tensor], c: Optional[StreamWeights]) -> None:
    T, S, W = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and S <= MAX_STREAMS
    assert (y is None) == (c is None) and (y is None or (y.shape == (T, W) and y.stride(1) == 1))


def hyper_step(x: torch.Tensor, y: Optional[torch.Tensor], c: Optional[StreamWeights], nxt: Optional[NextNorm], eps: float,
               act_dtype: torch.dtype) -> Normed:
    """x: fp32 streams [T, S, W], updated in place with the sublayer output y ([T, W], bf16 or fp32) and its stream weights (both
    None: unchanged).  Returns the next sublayer's input (in ``act_dtype``, fp32 or None); ``nxt`` None: neither."""
    _check(x, y, c)
    T, S, W = x.shape
    if x.is_cuda:
        out, out32 = _outputs(T, W, act_dtype, nxt, x.device)
        native.call("llmctl_hyper_step", x.data_ptr(), S, native.ptr(y), _is32(y) if y is not None else 0, y.stride(0) if y is not None else 0,
                    native.ptr(c.mix) if c else None, native.ptr(c.b) if c else None, native.ptr(nxt.a) if nxt else None,
                    native.ptr(nxt.w) if nxt else None, native.ptr(nxt.bias) if nxt else None, native.ptr(out), int(act_dtype == torch.float32),
                    native.ptr(out32), None, T, W, float(eps), native.stream_ptr())
        return _pair(out, out32, nxt)
    if y is not None:
        x.copy_(torch.einsum("nsw,st->ntw", x, c.mix) + c.b[None, :, None] * y.float()[:, None, :])
    if nxt is None:
        return None, None
    return _norm_cpu(x.sum(1) if nxt.a is None else torch.einsum("nsw,s->nw", x, nxt.a), nxt, eps, act_dtype)


def hyper_output(x: torch.Tensor, y: Optional[torch.Tensor], c: Optional[StreamWeights], rows: torch.Tensor, nxt: NextNorm, eps: float,
                 act_dtype: torch.dtype) -> torch.Tensor:
    """The normed sum [len(rows), W] of the selected rows' streams after the update; the streams themselves are not written."""
    _check(x, y, c)
    T, S, W = x.shape
    n = rows.numel()
    if x.is_cuda:
        out = torch.empty(n, W, dtype=act_dtype, device=x.device)
        native.call("llmctl_hyper_step", x.data_ptr(), S, native.ptr(y), _is32(y) if y is not None else 0, y.stride(0) if y is not None else 0,
                    native.ptr(c.mix) if c else None, native.ptr(c.b) if c else None, native.ptr(nxt.a), nxt.w.data_ptr(), nxt.bias.data_ptr(),
                    out.data_ptr(), int(act_dtype == torch.float32), None, rows.data_ptr(), n, W, float(eps), native.stream_ptr())
        return out
    xs = x[rows].clone()
    return hyper_step(xs, y[rows] if y is not None else None, c, nxt, eps, act_dtype)[0]
