"""Retention (linear attention with a fixed decay per head) over per-sequence state slots — csrc/recurrent/retention.cu.

``S <- decay_h S + k v^T;  o = S^T q`` per head on queries and keys whose first ``rot`` numbers are rotated by position (pairs
(i, i + rot/2)), keys scaled by ``d^(-1/2)``; every head's o is brought to unit RMS (no weight) and gated.  Portions, slots and
their reuse are as in ``ops/recurrent.py``; the state is ``[slots, H, d, e]`` fp32.

``retention`` is the whole mixer core between the projections and the output projection: for prompts a parallel prepare pass,
the scan and the head norm with its gate, or in bf16 (``uses_chunks``) chunks of 64 tokens as matrix products on the tensor
cores; for a batch in which every sequence decodes one token, one launch.  CPU tensors
run the PyTorch restatement below (CPU tests); on a GPU a missing kernel raises.

Reference: none — the reference has no model code (reference llmctl/runtime/engine.py:119-140)."""
from __future__ import annotations

import os
from typing import Optional

import torch

from . import native
from .elementwise import _is32, rotate_halves
from .matrix_state import MAX_DIM, _gate_kind, _pad_rows
from .recurrent import gla_output

c_void_p, c_int, c_ll, c_float = native.c_void_p, native.c_int, native.c_ll, native.c_float
native.register_signature("llmctl_retention_prepare", [c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_void_p, c_int, c_void_p, c_int,
                                                        c_void_p, c_int, c_int, c_int, c_int, c_void_p])
native.register_signature("llmctl_retention_scan", [c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p])
native.register_signature("llmctl_retention_step", [c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                                     c_int, c_void_p, c_void_p, c_ll, c_int, c_float, c_void_p, c_int, c_int, c_int, c_int,
                                                     c_void_p])

native.register_signature("llmctl_retention_chunked_ok", [c_int, c_int, c_int])
native.register_signature("llmctl_retention_chunked", [c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
                                                        c_int, c_void_p, c_int, c_int, c_void_p, c_void_p, c_ll, c_int, c_float, c_void_p, c_void_p,
                                                        c_int, c_void_p, c_int, c_int, c_int, c_void_p])
native._KERNELS_PER_CALL["llmctl_retention_chunked_ok"] = 0
native._KERNELS_PER_CALL["llmctl_retention_chunked"] = 4

CHUNK = 64                      # tokens per chunk
SCRATCH_NUMBERS = 64 << 20      # states kept between the chunked launches: heads are taken in passes of at most this many numbers


def uses_chunks(dtype: torch.dtype, d: int, e: int, rot: int) -> bool:
    """bf16 with d and e multiples of 16 up to 256 and rotated parts of a multiple of 8 numbers."""
    if dtype != torch.bfloat16 or not native.has_symbol("llmctl_retention_chunked"):
        return False
    if os.environ.get("LLMCTL_RETENTION", "") == "scan":        # ablation switch: the serial scan for bf16 too
        return False
    return bool(native.lib().llmctl_retention_chunked_ok(int(d), int(e), int(rot)))


def _aligned(*views: torch.Tensor) -> bool:
    return all(t.data_ptr() % 16 == 0 and t.stride(0) % 8 == 0 for t in views)


def retention_chunked(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, rot: int,
                      decay_m1: torch.Tensor, portions: torch.Tensor, tiles: torch.Tensor, state: torch.Tensor, H: int, d: int, e: int, eps: float,
                      gate_act: str) -> torch.Tensor:
    """Prompts in chunks (CUDA, bf16; arguments as in ``retention``): updates ``state``, returns the normed and gated output."""
    T, n = q.shape[0], tiles.shape[0]
    per_pass = max(1, min(H, SCRATCH_NUMBERS // max(n * d * e, 1)))
    cs = torch.empty(T, max(rot, 4), dtype=torch.float32, device=q.device)
    scratch = torch.empty(n * per_pass * d * e, dtype=torch.float32, device=q.device)
    out = torch.empty(T, H * e, dtype=q.dtype, device=q.device)
    native.call("llmctl_retention_chunked", q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), positions.data_ptr(),
                freq.data_ptr(), rot, decay_m1.data_ptr(), portions.data_ptr(), portions.shape[0], tiles.data_ptr(), n, T, state.data_ptr(),
                gate.data_ptr(), gate.stride(0), _gate_kind(gate_act), float(eps), cs.data_ptr(), scratch.data_ptr(), per_pass, out.data_ptr(), H, d, e,
                native.stream_ptr())
    return out


def work_numbers(tokens: int, H: int, d: int, e: int) -> int:
    """fp32 scratch of the prepare pass."""
    return tokens * H * (2 * _pad_rows(d) + (e + 31) // 32 * 32 + 4)


def retention_prepare(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, rot: int,
                      decay_m1: torch.Tensor, H: int, d: int, e: int) -> torch.Tensor:
    """The parallel pass before a scan (CUDA tensors, arguments as in ``retention``); returns the scan's scratch."""
    T = q.shape[0]
    work = torch.empty(work_numbers(T, H, d, e), dtype=torch.float32, device=q.device)
    native.call("llmctl_retention_prepare", q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), positions.data_ptr(),
                freq.data_ptr(), rot, decay_m1.data_ptr(), T, work.data_ptr(), H, d, e, _is32(q), native.stream_ptr())
    return work


def retention_scan(work: torch.Tensor, portions: torch.Tensor, state: torch.Tensor, T: int, H: int, d: int, e: int) -> torch.Tensor:
    """The serial pass over prepared tokens (CUDA tensors): updates ``state``, returns o, fp32 [T, H e]."""
    o = torch.empty(T, H * e, dtype=torch.float32, device=work.device)
    native.call("llmctl_retention_scan", work.data_ptr(), portions.data_ptr(), portions.shape[0], T, state.data_ptr(), o.data_ptr(), H, d, e,
                native.stream_ptr())
    return o


def retention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, rot: int,
              decay_m1: torch.Tensor, portions: torch.Tensor, state: torch.Tensor, H: int, d: int, e: int, eps: float, gate_act: str = "silu",
              decode: bool = False, tiles: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q, k: [T, H d]; v, gate: [T, H e] (gate: pre-activation), views with unit column stride of one type; freq: fp32 [rot / 2];
    decay_m1: fp32 [H], decay minus one (slow decays keep their precision).  ``decode``: every portion has one token;
    ``tiles``: the portions' tiles of 64 tokens (int32 [n, 4] = (first token row, tokens, portion, 0)), which allow the chunked
    form.  Updates
    ``state`` [slots, H, d, e] in place; returns ``o / rms(o) * act(gate)`` [T, H e] in the activations' type."""
    T = q.shape[0]
    assert d <= MAX_DIM and rot % 2 == 0 and rot <= d
    if q.is_cuda:
        assert all(t.stride(1) == 1 and t.dtype == q.dtype for t in (q, k, v, gate))
        assert state.is_contiguous() and state.dtype == torch.float32 and decay_m1.dtype == torch.float32
        if decode:
            out = torch.empty(T, H * e, dtype=q.dtype, device=q.device)
            native.call("llmctl_retention_step", q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), positions.data_ptr(),
                        freq.data_ptr(), rot, decay_m1.data_ptr(), portions.data_ptr(), portions.shape[0], state.data_ptr(), gate.data_ptr(),
                        gate.stride(0), _gate_kind(gate_act), float(eps), out.data_ptr(), H, d, e, _is32(q), native.stream_ptr())
            return out
        if tiles is not None and uses_chunks(q.dtype, d, e, rot) and _aligned(q, k, v, gate):
            return retention_chunked(q, k, v, gate, positions, freq, rot, decay_m1, portions, tiles, state, H, d, e, eps, gate_act)
        o = retention_scan(retention_prepare(q, k, v, positions, freq, rot, decay_m1, H, d, e), portions, state, T, H, d, e)
        return gla_output(o, None, gate, H, e, eps, q.dtype, gate_act)
    qf, kf, vf = q.float().reshape(T, H, d), k.float().reshape(T, H, d), v.float().reshape(T, H, e)
    if rot:
        qf, kf = (torch.cat([rotate_halves(t[..., :rot], positions[:T], freq), t[..., rot:]], dim=-1) for t in (qf, kf))
    kf = kf * d ** -0.5
    g = (1.0 + decay_m1.double()).float()[:, None, None]
    out = torch.zeros(T, H, e)
    for t0, n, pos0, slot in portions.tolist():
        if n <= 0:
            continue
        S = state[slot].clone() if (slot >= 0 and pos0 > 0) else torch.zeros(H, d, e)
        for t in range(t0, t0 + n):
            S = g * S + kf[t][:, :, None] * vf[t][:, None, :]
            out[t] = torch.einsum("hde,hd->he", S, qf[t])
        if slot >= 0:
            state[slot] = S
    return gla_output(out.reshape(T, H * e), None, gate, H, e, eps, q.dtype, gate_act)
