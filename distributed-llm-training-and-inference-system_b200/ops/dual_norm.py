"""Residual update and the two weighted RMS pre-norms of a parallel layer, and the embedding with sinusoidal positions —
csrc/norm/dual_norm.cu.

``residual_dual_norm``: ``x += m + f [+ add]`` on the fp32 stream and, from the same pass, ``w_s x / rms(x)`` for the next
layer's mixer and feed-forward.  The mixer's output is one tensor, or a ``BranchSum`` of two that are normed over the model
width before they join.  ``embed_sinusoid``: ``scale * table[token]`` plus sines and cosines of position times frequency.
CPU tensors run the PyTorch restatements below (CPU tests); on a GPU a missing kernel raises.

Reference: none — the reference has no model code (reference llmctl/runtime/engine.py:119-140)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple, Union

import torch

from . import native
from .elementwise import _is32

c_void_p, c_int, c_ll, c_float = native.c_void_p, native.c_int, native.c_ll, native.c_float
native.register_signature("llmctl_residual_dual_norm", [c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_void_p, c_float, c_void_p, c_ll, c_void_p,
                                                         c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_int,
                                                         c_void_p])
native.register_signature("llmctl_embed_sinusoid", [c_void_p, c_void_p, c_void_p, c_int, c_float, c_void_p, c_void_p, c_void_p, c_int, c_int,
                                                     c_void_p])


@dataclass
class BranchSum:
    """A mixer output ``factor * (wa a / rms(a) + wb b / rms(b))``: a, b [T, W] in the activation type, wa, wb fp32 [W]."""
    a: torch.Tensor
    b: torch.Tensor
    wa: torch.Tensor
    wb: torch.Tensor
    factor: float = 0.5


def sinusoid_frequencies(width: int, base: float = 10000.0) -> torch.Tensor:
    """``base^(-2 i / width)`` for the i-th (sine, cosine) pair, fp64 [(width + 1) // 2]."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / width)


def embed_sinusoid(tokens: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, scale: float, freq: torch.Tensor,
                   want_copy: bool = False) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``x[t] = scale * table[tokens[t]] + (sin at even, cos at odd columns of positions[t] * freq)``: (fp32 [T, W], a second
    copy or None)."""
    T, W = tokens.numel(), table.shape[1]
    if table.is_cuda:
        x = torch.empty(T, W, dtype=torch.float32, device=table.device)
        copy = torch.empty_like(x) if want_copy else None
        native.call("llmctl_embed_sinusoid", tokens.data_ptr(), positions.data_ptr(), table.data_ptr(), _is32(table), float(scale),
                    freq.data_ptr(), x.data_ptr(), native.ptr(copy), T, W, native.stream_ptr())
        return x, copy
    ang = positions.reshape(-1).to(torch.float64)[:, None] * freq
    pe = torch.stack([torch.sin(ang), torch.cos(ang)], dim=-1).flatten(1)[:, :W].float()
    x = table[tokens.reshape(-1)].float() * scale + pe
    return x, (x.clone() if want_copy else None)


def residual_dual_norm(m: Union[torch.Tensor, BranchSum, None], f: Optional[torch.Tensor], x: torch.Tensor, eps: float,
                       norm_w: Sequence[torch.Tensor], out_dtype: torch.dtype, add: Optional[torch.Tensor] = None) -> List[torch.Tensor]:
    """``x += m + f`` and then ``x += add`` in place on the fp32 stream [T, W] (each part optional; m and f in ``out_dtype`` with unit
    column stride, add fp32); returns ``w x / sqrt(mean(x^2) + eps)`` in ``out_dtype`` for each of the (up to two) fp32 weights."""
    T, W = x.shape
    S = len(norm_w)
    assert x.dtype == torch.float32 and x.is_contiguous() and S <= 2
    pair = isinstance(m, BranchSum)
    a, b = (m.a, m.b) if pair else (m, None)
    for t in (a, b, f):
        assert t is None or (t.shape == x.shape and t.stride(1) == 1 and t.dtype == out_dtype)
    assert add is None or (add.dtype == torch.float32 and add.is_contiguous() and add.shape == x.shape)
    if x.is_cuda:
        outs = [torch.empty(T, W, dtype=out_dtype, device=x.device) for _ in range(S)]
        native.call("llmctl_residual_dual_norm", native.ptr(a), a.stride(0) if a is not None else 0, native.ptr(b),
                    b.stride(0) if b is not None else 0, m.wa.data_ptr() if pair else None, m.wb.data_ptr() if pair else None,
                    float(m.factor) if pair else 1.0, native.ptr(f), f.stride(0) if f is not None else 0, native.ptr(add), x.data_ptr(), S,
                    norm_w[0].data_ptr() if S > 0 else None, outs[0].data_ptr() if S > 0 else None,
                    norm_w[1].data_ptr() if S > 1 else None, outs[1].data_ptr() if S > 1 else None, T, W, float(eps),
                    int(out_dtype == torch.float32), native.stream_ptr())
        return outs

    def rms(v: torch.Tensor) -> torch.Tensor:
        return v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)
    if pair:
        x += m.factor * (rms(a.float()) * m.wa + rms(b.float()) * m.wb) + (f.float() if f is not None else 0.0)
    elif a is not None or f is not None:
        x += (a.float() if a is not None else 0.0) + (f.float() if f is not None else 0.0)
    if add is not None:
        x += add
    n = rms(x)
    return [(n * w).to(out_dtype) for w in norm_w]
