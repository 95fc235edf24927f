"""Recurrences with a matrix state per head over per-sequence state slots — csrc/recurrent/matrix_state.cu.

Gated delta rule (``kind`` 0: one decay per head, 1: one per head and key row): q, k, v pass a short causal convolution and
silu, q and k become unit vectors; ``S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q``.
Decayed outer products with a bonus for the current token (``kind`` 2): ``o = S^T r + (sum r u k) v;  S <- diag(w) S + k v^T``
over inputs mixed with the previous token's (``token_shift``).

Portions, slots and their reuse are as in ``ops/recurrent.py``: int32 ``[n, 4] = (first token row, tokens, position of the first
token, state slot)``; position 0 starts from zeros whatever the slot holds; slot -1 keeps nothing.  A sequence's state is S
(``[slots, H, d, e]`` fp32) and the last raw rows that the next portion needs: ``taps - 1`` rows of the convolution's inputs,
or the previous token's row.

``delta_rule`` and ``bonus_memory`` are the whole mixer core between the projections and the output projection: for prompts a
parallel prepare pass, the serial scan and the head norm with its gate; for a batch in which every sequence decodes one
token, one launch.  CPU tensors run the PyTorch restatements below (CPU tests); on a GPU a missing kernel raises.

Reference: none — the reference has no model code (reference llmctl/runtime/engine.py:119-140)."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F

from . import native
from .elementwise import _is32
from .recurrent import gla_output

c_void_p, c_int, c_ll, c_float = native.c_void_p, native.c_int, native.c_ll, native.c_float
native.register_signature("llmctl_delta_prepare", [c_void_p, c_ll, c_void_p, c_void_p, c_int, c_void_p, c_ll, c_void_p, c_void_p, c_void_p, c_ll,
                                                    c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p])
native.register_signature("llmctl_bonus_prepare", [c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_void_p, c_int,
                                                    c_void_p, c_int, c_int, c_int, c_void_p])
native.register_signature("llmctl_matrix_scan", [c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p,
                                                  c_ll, c_int, c_int, c_void_p, c_int, c_void_p])
native.register_signature("llmctl_matrix_step", [c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_ll, c_void_p, c_void_p, c_int,
                                                  c_void_p, c_ll, c_void_p, c_void_p, c_void_p, c_void_p, c_ll, c_void_p, c_int, c_void_p,
                                                  c_void_p, c_int, c_void_p, c_ll, c_int, c_float, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                                  c_int, c_void_p])
native.register_signature("llmctl_token_shift", [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p])

DELTA_PER_HEAD, DELTA_PER_CHANNEL, BONUS = 0, 1, 2
MAX_DIM = 256           # key rows of a head


def _pad_rows(d: int) -> int:
    return 32 if d <= 32 else 64 if d <= 64 else 128 if d <= 128 else 256


def work_numbers(tokens: int, H: int, G: int, d: int, e: int, kind: int) -> int:
    """fp32 scratch of the prepare pass (same rule as llmctl_matrix_scan_work)."""
    dp, ep = _pad_rows(d), (e + 31) // 32 * 32
    return tokens * (2 * G * dp + H * ep + 4 * H + (H * dp if kind != DELTA_PER_HEAD else 0))


def _gate_kind(act: str) -> int:
    return {"silu": 0, "sigmoid": 1}[act]


def delta_prepare(qkv: torch.Tensor, conv_w: torch.Tensor, z: torch.Tensor, dt_bias: torch.Tensor, speed: torch.Tensor, b: torch.Tensor,
                  portions: torch.Tensor, seq_rows: torch.Tensor, conv_state: torch.Tensor, H: int, G: int, d: int, e: int,
                  kind: int) -> torch.Tensor:
    """The parallel pass before a delta-rule scan (CUDA tensors, arguments as in ``delta_rule``); returns the scan's scratch."""
    T, taps = qkv.shape[0], conv_w.shape[1]
    work = torch.empty(work_numbers(T, H, G, d, e, kind), dtype=torch.float32, device=qkv.device)
    native.call("llmctl_delta_prepare", qkv.data_ptr(), qkv.stride(0), conv_w.data_ptr(), conv_state.data_ptr() if taps > 1 else None, taps,
                z.data_ptr(), z.stride(0), dt_bias.data_ptr(), speed.data_ptr(), b.data_ptr(), b.stride(0), portions.data_ptr(),
                seq_rows.data_ptr(), T, work.data_ptr(), H, G, d, e, kind, _is32(qkv), native.stream_ptr())
    return work


def bonus_prepare(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, z: torch.Tensor, w0: torch.Tensor, u: torch.Tensor, H: int,
                  d: int) -> torch.Tensor:
    """The parallel pass before a bonus-memory scan (CUDA tensors, arguments as in ``bonus_memory``); returns the scan's scratch."""
    T = r.shape[0]
    work = torch.empty(work_numbers(T, H, H, d, d, BONUS), dtype=torch.float32, device=r.device)
    native.call("llmctl_bonus_prepare", r.data_ptr(), r.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), z.data_ptr(), z.stride(0),
                w0.data_ptr(), u.data_ptr(), T, work.data_ptr(), H, d, _is32(r), native.stream_ptr())
    return work


def matrix_scan(work: torch.Tensor, portions: torch.Tensor, state: torch.Tensor, T: int, H: int, G: int, d: int, e: int, kind: int,
                tail: torch.Tensor, tail_state: torch.Tensor) -> torch.Tensor:
    """The serial pass over prepared tokens (CUDA tensors): updates ``state``, stores the last rows of ``tail`` [T, C] into
    ``tail_state`` [slots, keep, C] and returns o, fp32 [T, H e]."""
    o = torch.empty(T, H * e, dtype=torch.float32, device=work.device)
    keep = tail_state.shape[1]
    native.call("llmctl_matrix_scan", work.data_ptr(), portions.data_ptr(), portions.shape[0], T, state.data_ptr(), o.data_ptr(), H, G, d, e, kind,
                tail.data_ptr(), tail.stride(0), tail.shape[1], keep, tail_state.data_ptr() if keep else None, _is32(tail),
                native.stream_ptr())
    return o


def delta_rule(qkv: torch.Tensor, conv_w: torch.Tensor, z: torch.Tensor, dt_bias: torch.Tensor, speed: torch.Tensor, b: torch.Tensor,
               gate: torch.Tensor, norm_w: torch.Tensor, portions: torch.Tensor, seq_rows: torch.Tensor, state: torch.Tensor,
               conv_state: torch.Tensor, H: int, G: int, d: int, e: int, per_channel: bool, eps: float, gate_act: str,
               decode: bool = False) -> torch.Tensor:
    """qkv: [T, 2 G d + H e] raw projections; conv_w: fp32 [2 G d + H e, taps] (last column = the current token's); z: decay
    projection, [T, H d] if ``per_channel`` else [T, H], with dt_bias alike (fp32) and speed = exp(A_log) (fp32 [H]); b: [T, H] write-strength logits;
    gate: [T, H e] pre-activation; norm_w: fp32 [e].  All activations are views with unit column stride of one type.
    ``decode``: every portion has one token.  Updates ``state`` [slots, H, d, e] and ``conv_state`` [slots, taps - 1, C] in
    place; returns ``rms-norm(o) * norm_w * act(gate)`` [T, H e] in the activations' type."""
    T, C = qkv.shape
    taps = conv_w.shape[1]
    kind = DELTA_PER_CHANNEL if per_channel else DELTA_PER_HEAD
    assert C == 2 * G * d + H * e and H % G == 0 and d <= MAX_DIM and z.shape[1] == dt_bias.numel() == (H * d if per_channel else H)
    if qkv.is_cuda:
        assert all(t.stride(1) == 1 and t.dtype == qkv.dtype for t in (qkv, z, b, gate))
        assert state.is_contiguous() and conv_state.is_contiguous() and conv_w.is_contiguous() and state.dtype == torch.float32
        cs = conv_state.data_ptr() if taps > 1 else None
        if decode:
            out = torch.empty(T, H * e, dtype=qkv.dtype, device=qkv.device)
            native.call("llmctl_matrix_step", qkv.data_ptr(), qkv.stride(0), None, 0, None, 0, None, 0, conv_w.data_ptr(), cs, taps, z.data_ptr(),
                        z.stride(0), dt_bias.data_ptr(), speed.data_ptr(), None, b.data_ptr(), b.stride(0), portions.data_ptr(),
                        portions.shape[0], state.data_ptr(), norm_w.data_ptr(), 0, gate.data_ptr(), gate.stride(0), _gate_kind(gate_act),
                        float(eps), out.data_ptr(), H, G, d, e, kind, _is32(qkv), native.stream_ptr())
            return out
        work = delta_prepare(qkv, conv_w, z, dt_bias, speed, b, portions, seq_rows, conv_state, H, G, d, e, kind)
        o = matrix_scan(work, portions, state, T, H, G, d, e, kind, qkv, conv_state)
        return gla_output(o, norm_w, gate, H, e, eps, qkv.dtype, gate_act)
    rep = H // G
    xf, keep = qkv.float(), taps - 1
    zt = F.softplus(z.float() + dt_bias)
    g = torch.exp(-(speed[:, None] * (zt.view(T, H, d) if kind == DELTA_PER_CHANNEL else zt.view(T, H, 1))))      # [T, H, d or 1]
    beta = torch.sigmoid(b.float())
    out = torch.zeros(T, H, e)
    for t0, n, pos0, slot in portions.tolist():
        if n <= 0:
            continue
        cont = slot >= 0 and pos0 > 0
        rows = torch.cat([conv_state[slot] if cont else torch.zeros(keep, C), xf[t0:t0 + n]], dim=0)
        y = F.silu(sum(rows[j:j + n] * conv_w[:, j] for j in range(taps)))
        q, k = y[:, :G * d].reshape(n, G, d), y[:, G * d:2 * G * d].reshape(n, G, d)
        q, k = (v / torch.sqrt(v.pow(2).sum(-1, keepdim=True) + 1e-6) for v in (q, k))
        q, k = (q * d ** -0.5).repeat_interleave(rep, dim=1), k.repeat_interleave(rep, dim=1)                       # [n, H, d]
        v = y[:, 2 * G * d:].reshape(n, H, e)
        S = state[slot].clone() if cont else torch.zeros(H, d, e)
        for i in range(n):
            S = g[t0 + i][:, :, None] * S
            u = beta[t0 + i][:, None] * (v[i] - torch.einsum("hde,hd->he", S, k[i]))
            S = S + k[i][:, :, None] * u[:, None, :]
            out[t0 + i] = torch.einsum("hde,hd->he", S, q[i])
        if slot >= 0:
            state[slot] = S
            if keep:
                conv_state[slot] = rows[-keep:]
    return gla_output(out.reshape(T, H * e), norm_w, gate, H, e, eps, qkv.dtype, gate_act)


def bonus_memory(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, z: torch.Tensor, w0: torch.Tensor, u: torch.Tensor, gate: torch.Tensor,
                 norm_w: torch.Tensor, h: torch.Tensor, portions: torch.Tensor, state: torch.Tensor, shift_state: torch.Tensor, H: int,
                 d: int, eps: float, gate_act: str = "silu", decode: bool = False) -> torch.Tensor:
    """r, k, v, z, gate: [T, H d] (views with unit column stride of one type; z: decay projection, the decay is
    ``exp(-exp(z + w0))``; gate: pre-activation); w0, u: fp32 [H d]; norm_w: fp32 [H d]; h: [T, W] contiguous, the token-shifted
    stream whose last row the next portion needs (``token_shift`` has stored it already for portions of one token).  Updates
    ``state`` [slots, H, d, d] and ``shift_state`` [slots, W] in place; returns ``rms-norm(o) * norm_w * act(gate)``."""
    T, W = h.shape
    assert d <= MAX_DIM
    if r.is_cuda:
        assert all(t.stride(1) == 1 and t.dtype == r.dtype for t in (r, k, v, z, gate, h)) and h.is_contiguous()
        assert state.is_contiguous() and shift_state.is_contiguous() and state.dtype == torch.float32
        if decode:
            out = torch.empty(T, H * d, dtype=r.dtype, device=r.device)
            native.call("llmctl_matrix_step", None, 0, r.data_ptr(), r.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), None, None,
                        1, z.data_ptr(), z.stride(0), w0.data_ptr(), None, u.data_ptr(), None, 0, portions.data_ptr(), portions.shape[0],
                        state.data_ptr(), norm_w.data_ptr(), d, gate.data_ptr(), gate.stride(0), _gate_kind(gate_act), float(eps),
                        out.data_ptr(), H, H, d, d, BONUS, _is32(r), native.stream_ptr())
            return out
        work = bonus_prepare(r, k, v, z, w0, u, H, d)
        o = matrix_scan(work, portions, state, T, H, H, d, d, BONUS, h, shift_state[:, None])
        return gla_output(o, norm_w, gate, H, d, eps, r.dtype, gate_act)
    w = torch.exp(-torch.exp(z.float() + w0)).view(T, H, d)
    rf, kf, vf, uf = r.float().reshape(T, H, d), k.float().reshape(T, H, d), v.float().reshape(T, H, d), u.view(H, d)
    out = torch.zeros(T, H, d)
    for t0, n, pos0, slot in portions.tolist():
        if n <= 0:
            continue
        S = state[slot].clone() if (slot >= 0 and pos0 > 0) else torch.zeros(H, d, d)
        for t in range(t0, t0 + n):
            kv = kf[t][:, :, None] * vf[t][:, None, :]
            out[t] = torch.einsum("hde,hd->he", S + uf[:, :, None] * kv, rf[t])
            S = w[t][:, :, None] * S + kv
        if slot >= 0:
            state[slot] = S
            shift_state[slot] = h[t0 + n - 1].float()
    return gla_output(out.reshape(T, H * d), norm_w, gate, H, d, eps, r.dtype, gate_act)


def token_shift(h: torch.Tensor, mu: torch.Tensor, portions: torch.Tensor, seq_rows: torch.Tensor, shift_state: torch.Tensor,
                out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[s, t] = h[t] + (h[t - 1] - h[t]) * mu[s]``; h: contiguous [T, W]; mu: fp32 [n, W]; shift_state: fp32 [slots, W], the row
    before each portion (zeros at position 0).  Returns [n, T, W] in h's type.  A portion of one token also stores its row;
    longer portions leave that to ``bonus_memory``."""
    T, W = h.shape
    n = mu.shape[0]
    if h.is_cuda:
        assert h.is_contiguous() and mu.is_contiguous() and mu.dtype == torch.float32 and shift_state.is_contiguous()
        out = torch.empty(n, T, W, dtype=h.dtype, device=h.device) if out is None else out
        native.call("llmctl_token_shift", h.data_ptr(), mu.data_ptr(), n, portions.data_ptr(), seq_rows.data_ptr(), shift_state.data_ptr(),
                    out.data_ptr(), T, W, _is32(h), native.stream_ptr())
        return out
    hf = h.float()
    prev = torch.zeros(T, W)
    for t0, cnt, pos0, slot in portions.tolist():
        if cnt <= 0:
            continue
        if slot >= 0 and pos0 > 0:
            prev[t0] = shift_state[slot]
        prev[t0 + 1:t0 + cnt] = hf[t0:t0 + cnt - 1]
        if slot >= 0 and cnt == 1:
            shift_state[slot] = hf[t0]
    return (hf + (prev - hf) * mu[:, None, :]).to(h.dtype)
