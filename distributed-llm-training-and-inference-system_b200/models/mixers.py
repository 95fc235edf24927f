"""Sequence mixers for ragged, paged inference batches.

``LatentAttention``: attention whose keys and values are linear images of one cached low-rank latent per token plus a
single rotated key part shared by all heads.  Queries go through their own normed latent.  Only ``[c | kr]`` is cached
(``R + dr`` numbers per token and layer instead of ``2 H d``); a layer may also read the cache of an earlier layer
(``kv_from``) and then has no key/value down-projection at all.  Per step:

    d        = h Wd^T                (one packed GEMM: query latent | key/value latent | key rope part)
    cq, cache= norm / rotate / append        (ops.latent_attention.latent_kv_write)
    q        = cq Wuq^T              [T, H, dn + dr]
    ql       = qn Uk_h               [T, H, R]   absorbed queries, fp32
    ol       = attention over the cache rows (ops.latent_attention.latent_attention)   [T, H, R]
    out      = (ol Uv_h^T) Wo^T

Optional parts of ``LatentAttention`` (fields of its spec): ``sink`` — a learned number per head whose exponential joins
the softmax denominator (a key without a value, not scaled); ``out_gate`` — the concatenated heads are multiplied element
by element with the sigmoid of one more projection of the mixer's input (packed into the down-projection GEMM);
``head_gate`` — the same with one number per head, applied by the attention kernel; ``window`` — a token sees itself and the
``window - 1`` tokens before it.  ``q_rank`` 0: queries are projected from the mixer's input directly (in the same packed
GEMM), ``rot_dim`` 0: no rotated part.

``SoftcapWindowAttention``: grouped-query attention whose scores pass a tanh soft cap and lose a linear
distance bias with one slope per head; a sliding window that also keeps the first tokens of the sequence; chunks (a query
sees the keys of its own chunk only); a softmax with one added to the denominator (a sink of score 0) or with a learned
sink per head; an RMS norm over the whole q and k projections and rotation of the first ``rot_dims`` numbers of every head
(pairs (i, i + rot_dims/2)); values cached at unit RMS per head; projection biases; a sigmoid output
gate; queries and keys at unit RMS per head; a query temperature that grows with the position; a learned bias per
logarithmic distance bucket.  Every part is a field of ``SoftcapWindowAttentionSpec``.  Per step:

    p        = h Wp^T                           (one packed GEMM: q | k | v | gate)
    q, cache = bias / value norm / append       (ops.softcap_attention.window_kv_append, or with projection norms or
                                                 rotation ops.window_attention.window_qkv_write)
    o        = attention over kept + window keys, gate      (ops.softcap_attention.softcap_window_attention)
    out      = o Wo^T + bo

``PooledWindowAttention``: grouped-query attention over a sliding window of ``window`` tokens plus one pooled key/value
(the mean of the cached keys / values) per block of ``pool`` tokens that lies wholly before the window.  Optional parts,
each a field of ``PooledWindowAttentionSpec``: projection biases, an RMS norm over the whole q and the whole k
projection, rotation of the first ``rot_dims`` numbers of every head (plain or YaRN-blended spectrum), a learned score
temperature per head, mixing of the normalised attention weights across heads by a learned [H, H] matrix, and mixing of
the layer's values with the values the first such layer computed for the same token.  Per step:

    qkv      = h Wqkv^T                         (one packed GEMM)
    q, cache = bias / norm / rotate / value mix / append     (ops.window_attention.window_qkv_write)
    pooled rows of the blocks the step completes             (ops.window_attention.window_pool_update)
    o        = attention over window + pooled rows           (ops.window_attention.pooled_window_attention)
    out      = o Wo^T

``DifferentialAttention``: grouped-query attention in which every head has two score maps (two query vectors against
two key vectors of its key/value head) over the same values; the head's output is ``a1 - lam a2`` brought to unit RMS,
times ``1 - diff`` and, optionally, a sigmoid gate per (token, head).  ``lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff`` is
one number of the layer.  Partial interleaved rotation on every query and key vector.  Per step:

    p        = h Wp^T                           (one packed GEMM: q | k | v | gate logits)
    q, cache = rotate / append                  (ops.diff_attention.rotary_kv_append)
    o        = both maps, difference, norm, gate        (ops.diff_attention.diff_attention)
    out      = o Wo^T

``GatedLinearAttention`` and ``SelectiveScan`` are recurrences: they keep no per-token cache but ONE state per sequence
in a state slot (``serve/ragged.py`` ``RaggedBatch.portions`` names each portion's slot), fp32.

``GatedLinearAttention``: per head ``S <- diag(a) S + k v^T``, ``o = S^T q`` with a decay per key channel
``a = sigmoid(z)^(1/tau)``, ``z`` from a low-rank projection with bias; heads are RMS-normed with one shared weight,
gated by ``silu`` of a projection and projected out.  Per step: one packed GEMM (q | k | v | gate | decay latent), the small
decay GEMM, ``ops.recurrent.gla_scan``, ``ops.recurrent.gla_output``, the output GEMM.

``SelectiveScan`` (Mamba): ``[x | z] = h Win^T``; ``u = silu(causal conv(x))``; ``[dt | B | C] = u Wx^T``;
``dt = softplus(dt Wdt^T + b)``; ``S <- exp(dt A) S + dt u B``, ``y = (S C + D u) silu(z)``; output GEMM.  The state of a
sequence is S and the last ``taps - 1`` inputs of the convolution.

``DeltaRule``: gated delta rule with a matrix state per head.  q, k, v pass a short causal convolution and silu, q and k become
unit vectors; ``S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q`` with one decay per head, or one per head and key row
from a low-rank projection; heads are RMS-normed with one shared weight and gated (sigmoid of a low-rank projection, or silu
of a full one).  Per step: one packed GEMM (q | k | v | latents or gate and decay | write strength), one block-diagonal GEMM for
both low-rank projections, ``ops.matrix_state.delta_rule``, the output GEMM.

``BonusMemory`` (RWKV-style time mixing): every projection reads its own mix of the token's and the previous token's input;
``o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T`` with a data-dependent decay per key row; heads RMS-normed, times a weight
and a silu gate.  Per step: ``ops.matrix_state.token_shift``, one batched GEMM (r, k, v, gate), the low-rank decay (two GEMMs and
a tanh), ``ops.matrix_state.bonus_memory``, the output GEMM.

``Retention``: ``S <- decay_h S + k v^T,  o = S^T q`` with a fixed decay per head on rotated queries and keys; heads brought to
unit RMS and gated by silu of a projection.  Per step: one packed GEMM (q | k | v | gate), ``ops.retention.retention``, the
output GEMM.

``BranchPair``: two mixers side by side on one input; its output is an ``ops.dual_norm.BranchSum`` that the residual update
evaluates (each branch RMS-normed over the model width with a weight of its own, half their sum).

Reference: none — the reference has no model code (reference llmctl/runtime/engine.py:119-140)."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

import torch
import torch.nn as nn

from ..ops import diff_attention as dops
from ..ops import functional as ops
from ..ops import latent_attention as lops
from ..ops import matrix_state as mops
from ..ops import recurrent as rops
from ..ops import retention as retops
from ..ops import softcap_attention as sops
from ..ops import window_attention as wops
from ..ops.dual_norm import BranchSum
from ..ops.elementwise import rope_frequencies, sigmoid_gate_, tanh_


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class LatentAttentionSpec:
    heads: int
    dim: int            # unrotated query/key size per head (dn)
    rot_dim: int        # rotated query/key size per head (dr)
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_base: float
    rot_scaling: Optional[Dict[str, Any]] = None
    kv_from: Optional[int] = None       # index of the layer whose cache this layer reads
    sink: bool = False                  # a learned number per head joins the softmax denominator
    out_gate: bool = False              # heads * sigmoid(Wg h) before the output projection
    head_gate: bool = False             # the same with one gate per head
    window: int = 0                     # a token sees itself and the window - 1 tokens before it; 0: every earlier token

    @property
    def cache_width(self) -> int:
        return self.kv_rank + self.rot_dim


class LatentAttention(nn.Module):
    stateful = False

    def __init__(self, width: int, spec: LatentAttentionSpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        self.eps = eps
        own = s.kv_from is None
        if (s.out_gate and s.head_gate) or s.window < 0 or (s.q_rank == 0 and not own):
            raise ValueError(f"inconsistent latent attention parts: {s}")
        kw = dict(dtype=dtype, device=device)
        self.n_down = s.q_rank + (s.kv_rank + s.rot_dim if own else 0)
        # rows of the packed projection: [dq ; dkv ; gate], or without a query latent [dkv ; q ; gate], those parts starting at
        # multiples of 8
        self.q_at = 0 if s.q_rank else _pad8(self.n_down)
        self.gate_at = self.n_down if s.q_rank else self.q_at + _pad8(s.heads * (s.dim + s.rot_dim))
        n_gate = s.heads * s.vdim if s.out_gate else s.heads if s.head_gate else 0
        rows = self.gate_at + n_gate
        self.w_down = nn.Parameter(torch.zeros(rows if s.q_rank else _pad8(rows), width, **kw))
        self.sink = nn.Parameter(torch.zeros(s.heads, dtype=torch.float32, device=device)) if s.sink else None
        self.q_norm = nn.Parameter(torch.ones(s.q_rank, **kw)) if s.q_rank else None
        self.kv_norm = nn.Parameter(torch.ones(s.kv_rank, **kw)) if own else None
        self.w_uq = nn.Parameter(torch.empty(s.heads * (s.dim + s.rot_dim), s.q_rank, **kw)) if s.q_rank else None
        self.w_uk = nn.Parameter(torch.empty(s.heads, s.dim, s.kv_rank, **kw))          # per head [dn, R]
        self.w_uv = nn.Parameter(torch.empty(s.heads, s.vdim, s.kv_rank, **kw))         # per head [dv, R]
        self.w_o = nn.Parameter(torch.empty(width, s.heads * s.vdim, **kw))
        f, self.rot_mult = rope_frequencies(s.rot_dim, s.rot_base, s.rot_scaling)
        self.register_buffer("rot_freq", f.to(device), persistent=False)

    def load(self, get, prefix: str) -> None:
        s = self.spec
        with torch.no_grad():
            parts = ([(0, "dq")] if s.q_rank else [(self.q_at, "q")]) + ([(s.q_rank, "dkv")] if s.kv_from is None else [])
            for at, name in parts + ([(self.gate_at, "g")] if s.out_gate or s.head_gate else []):
                w = get(prefix + name)
                self.w_down[at:at + w.shape[0]].copy_(w)
            if s.sink:
                self.sink.copy_(get(prefix + "sink").float())
            if s.q_rank:
                self.q_norm.copy_(get(prefix + "dq.norm"))
                self.w_uq.copy_(get(prefix + "uq"))
            if s.kv_from is None:
                self.kv_norm.copy_(get(prefix + "dkv.norm"))
            self.w_uk.copy_(get(prefix + "uk").view(s.heads, s.dim, s.kv_rank))
            self.w_uv.copy_(get(prefix + "uv").view(s.heads, s.vdim, s.kv_rank))
            self.w_o.copy_(get(prefix + "o"))

    def forward(self, h: torch.Tensor, batch, cache: torch.Tensor) -> torch.Tensor:
        """h: [T, W] in the activation type; ``cache``: this layer's (or its source layer's) [blocks, bs, R + dr]."""
        s = self.spec
        T = h.shape[0]
        own = s.kv_from is None
        d = ops.linear(h, self.w_down)
        cq = lops.latent_kv_write(d, s.q_rank, s.kv_rank if own else 0, s.rot_dim if own else 0, self.q_norm, self.kv_norm,
                                  cache if own else None, batch.slots, batch.positions, self.rot_freq, self.rot_mult, self.eps)
        nq = s.heads * (s.dim + s.rot_dim)
        q = ops.linear(cq, self.w_uq) if s.q_rank else d[:, self.q_at:self.q_at + nq]   # [T, H * (dn + dr)]
        qn = q.unflatten(1, (s.heads, s.dim + s.rot_dim))[:, :, :s.dim].transpose(0, 1) # [H, T, dn], a view
        # absorbed queries ql[t, h] = Uk_h^T qn[t, h]: fp32, except that the tensor-core attention kernel takes them
        # in bf16 (it multiplies in bf16 anyway); the kernel reads the [H, T, R] product through its strides
        if q.is_cuda and q.dtype == torch.bfloat16:
            if lops.uses_tensor_cores(q.dtype, s.kv_rank, s.rot_dim):
                ql = torch.bmm(qn, self.w_uk)
            else:
                ql = torch.bmm(qn, self.w_uk, out_dtype=torch.float32)
        else:
            ql = torch.bmm(qn.float(), self.w_uk.float())
        ql = ql.transpose(0, 1)
        # batches with prompt portions fill the tcgen05 kernel's 128-row tiles; a decoding token has only its heads to
        # offer, and the 16 / 32-row kernel reads the cache once for them
        if not batch.decode_only and lops.uses_tcgen05(q.dtype, s.kv_rank, s.rot_dim, cache.shape[1], q.is_cuda):
            rows = lops.ROWS_PER_TILE_TCGEN05
        else:
            rows = lops.rows_per_tile(q.dtype, s.kv_rank, s.rot_dim, q.is_cuda, s.heads if batch.decode_only else lops.ROWS_PER_TILE_WIDE)
        hpt = batch.heads_per_tile(s.heads, rows)
        span = lops.key_span(batch.max_context, s.window, rows // hpt)
        ol = lops.latent_attention(ql, q, s.dim, cache, batch.block_tables, batch.tiles(rows), batch.positions,
                                   self.rot_freq, self.rot_mult, s.scale, hpt, batch.max_context,
                                   batch.attention_splits(s.heads, rows, span), rows=rows, sinks=self.sink, window=s.window,
                                   head_gate=d[:, self.gate_at:self.gate_at + s.heads] if s.head_gate else None)
        o = torch.empty(T, s.heads * s.vdim, dtype=ol.dtype, device=ol.device)          # the product lands head by head in place
        with torch.no_grad():
            torch.bmm(ol.transpose(0, 1), self.w_uv.transpose(1, 2), out=o.view(T, s.heads, s.vdim).transpose(0, 1))
        if s.out_gate:
            o = sigmoid_gate_(o, d[:, self.gate_at:self.gate_at + s.heads * s.vdim])
        return ops.linear(o, self.w_o)

    def cache_shape(self, num_blocks: int, block_size: int) -> Tuple[int, ...]:
        return (num_blocks, block_size, self.spec.cache_width)


@dataclass
class PooledWindowAttentionSpec:
    heads: int
    kv_heads: int
    dim: int            # query/key size per head
    vdim: int           # value size per head
    scale: float
    window: int = 0     # 0: every earlier token is seen, nothing is pooled
    pool: int = 0       # tokens per pooled block
    rot_dims: int = 0   # rotated numbers per head (even, <= dim); 0: no rotation
    rot_base: float = 10000.0
    rot_scaling: Optional[Dict[str, Any]] = None
    bias: bool = True
    qk_norm: bool = True            # RMS norm over the whole q / k projection, per-coordinate weights
    head_temperature: bool = True   # scores of head h are multiplied by a learned number
    talking_heads: bool = True      # normalised weights are mixed across heads by a learned [H, H] matrix
    v_mix: bool = False             # values are blended with those of the first v_mix layer

    @property
    def cache_width(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)

    def rows_per_page(self, block_size: int) -> int:
        return block_size + wops.pooled_rows_per_page(block_size, self.pool if self.window else 0)


class PooledWindowAttention(nn.Module):
    TILE_TOKENS = 16        # tile width of the ragged batch this mixer asks for (serve/ragged.py)

    def __init__(self, width: int, spec: PooledWindowAttentionSpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        if s.heads % s.kv_heads or s.rot_dims % 2 or s.rot_dims > s.dim or (s.window and s.pool < 1):
            raise ValueError(f"inconsistent attention sizes: {s}")
        self.eps = eps
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        nq, nk, nv = s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim
        self.w_qkv = nn.Parameter(torch.empty(nq + nk + nv, width, **kw))               # [q ; k ; v]
        self.b_qkv = nn.Parameter(torch.zeros(nq + nk + nv, **kw)) if s.bias else None
        self.q_norm = nn.Parameter(torch.ones(nq, **f32)) if s.qk_norm else None
        self.k_norm = nn.Parameter(torch.ones(nk, **f32)) if s.qk_norm else None
        self.temp = nn.Parameter(torch.ones(s.heads, **f32)) if s.head_temperature else None
        self.talk = nn.Parameter(torch.eye(s.heads, **f32)) if s.talking_heads else None
        self.vmix = nn.Parameter(torch.zeros(1, **f32)) if s.v_mix else None
        self.w_o = nn.Parameter(torch.empty(width, s.heads * s.vdim, **kw))
        if s.rot_dims:
            f, self.rot_mult = rope_frequencies(s.rot_dims, s.rot_base, s.rot_scaling)
        else:
            f, self.rot_mult = torch.zeros(1), 1.0
        self.register_buffer("rot_freq", f.to(device), persistent=False)

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: q, k, v (+ ``.b`` biases, ``q.norm`` / ``k.norm``), temp, talk, vmix, o."""
        s = self.spec
        with torch.no_grad():
            self.w_qkv.copy_(torch.cat([get(prefix + "q"), get(prefix + "k"), get(prefix + "v")], dim=0))
            if s.bias:
                self.b_qkv.copy_(torch.cat([get(prefix + "q.b"), get(prefix + "k.b"), get(prefix + "v.b")], dim=0))
            if s.qk_norm:
                self.q_norm.copy_(get(prefix + "q.norm").float())
                self.k_norm.copy_(get(prefix + "k.norm").float())
            if s.head_temperature:
                self.temp.copy_(get(prefix + "temp").float())
            if s.talking_heads:
                self.talk.copy_(get(prefix + "talk").float())
            if s.v_mix:
                self.vmix.copy_(get(prefix + "vmix").float().reshape(1))
            self.w_o.copy_(get(prefix + "o"))

    def forward(self, h: torch.Tensor, batch, cache: torch.Tensor, v_first: Optional[torch.Tensor] = None):
        """h: [T, W] in the activation type; ``cache``: this layer's [pages, bs + PS, G (d + e)].  ``v_first``: the values
        of the first v_mix layer for the step's tokens (None in that layer itself, which then returns them).  Returns
        (output [T, W], v_first)."""
        s = self.spec
        T = h.shape[0]
        bs = batch.block_size
        qkv = ops.linear(h, self.w_qkv)
        v_mode = 0
        if s.v_mix:
            v_mode = 2 if v_first is not None else 1
            if v_first is None:
                v_first = torch.empty(T, s.kv_heads * s.vdim, dtype=h.dtype, device=h.device)
        q = wops.window_qkv_write(qkv, self.b_qkv, self.q_norm, self.k_norm, s.heads, s.kv_heads, s.dim, s.vdim, s.rot_dims,
                                  self.rot_freq, self.rot_mult, self.eps, batch.positions, batch.slots, cache, bs,
                                  v_first if v_mode else None, v_mode, self.vmix)
        pool = s.pool if s.window else 0
        wops.window_pool_update(cache, batch.positions, batch.slots, batch.seq_rows, batch.block_tables, bs, pool)
        o = wops.pooled_window_attention(q, cache, batch.block_tables, batch.tiles(self.TILE_TOKENS),
                                         1 if batch.decode_only else self.TILE_TOKENS, batch.positions, self.temp, self.talk,
                                         s.scale, s.heads, s.kv_heads, s.dim, s.vdim, s.window, pool, bs, h.dtype,
                                         max_context=batch.max_context)
        return ops.linear(o, self.w_o), v_first


@dataclass
class SoftcapWindowAttentionSpec:
    heads: int
    kv_heads: int
    dim: int            # query/key size per head
    vdim: int           # value size per head
    scale: float
    softcap: float = 0.0        # scores become softcap * tanh(score / softcap); 0: no cap
    window: int = 0             # position i sees j <= i with i - j < window; 0: every earlier token
    keep_first: int = 0         # ... or j < keep_first
    distance_bias: bool = True  # slope_h (i - j) is taken off the score, slope_h = 2^(-8 (h + 1) / heads)
    sink_one: bool = True       # one is added to the softmax denominator (a sink of score 0 without a value)
    value_norm: bool = True     # every value head is cached at unit RMS (no weight)
    bias: bool = True           # q, k, v and output projections have biases
    out_gate: bool = True       # heads * sigmoid(Wg h) before the output projection
    qk_norm: bool = False       # queries and keys are brought to unit RMS per head (no weight)
    q_temp: Optional[Tuple[float, float]] = None    # (coef, every): q *= 1 + coef ln(floor((p + 1) / every) + 1)
    bias_rows: int = 0          # rows of a learned bias per distance bucket and head (0: none)
    bias_max: float = 0.0       # distance at which the last bucket begins at the latest
    chunk: int = 0              # position i sees only keys of its own chunk of this many positions; 0: no chunks
    sink: bool = False          # a learned number per head joins the softmax denominator (instead of sink_one)
    proj_norm: bool = False     # RMS norm over the whole q and the whole k projection, per-coordinate weights
    rot_dims: int = 0           # rotated numbers per head, pairs (i, i + rot_dims/2); 0: no rotation
    rot_base: float = 10000.0
    out_bias: bool = True       # with ``bias``: the output projection has one too

    @property
    def cache_width(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)


class SoftcapWindowAttention(nn.Module):
    stateful = False

    def __init__(self, width: int, spec: SoftcapWindowAttentionSpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        if s.heads % s.kv_heads or s.window < 0 or s.keep_first < 0 or s.softcap < 0 or s.chunk < 0 or (s.sink and s.sink_one):
            raise ValueError(f"inconsistent attention sizes: {s}")
        # projection norms and rotation come with their own append kernel, which has no per-head norms and no temperature
        self.rotary_append = s.proj_norm or s.rot_dims > 0
        if self.rotary_append and (s.value_norm or s.qk_norm or s.q_temp or s.rot_dims % 2 or s.rot_dims > s.dim):
            raise ValueError(f"attention parts that do not go together: {s}")
        self.eps = eps
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        self.nq, self.nk, self.nv = s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim
        self.n_qkv = self.nq + self.nk + self.nv
        self.w_in = nn.Parameter(torch.empty(self.n_qkv + (s.heads * s.vdim if s.out_gate else 0), width, **kw))     # [q ; k ; v ; gate]
        self.b_in = nn.Parameter(torch.zeros(self.n_qkv, **f32)) if s.bias else None
        self.w_o = nn.Parameter(torch.empty(width, s.heads * s.vdim, **kw))
        self.b_o = nn.Parameter(torch.zeros(width, **f32)) if s.bias and s.out_bias else None
        self.q_norm = nn.Parameter(torch.ones(self.nq, **f32)) if s.proj_norm else None
        self.k_norm = nn.Parameter(torch.ones(self.nk, **f32)) if s.proj_norm else None
        self.register_buffer("rot_freq", rope_frequencies(s.rot_dims, s.rot_base)[0].to(device) if s.rot_dims else None, persistent=False)
        self.register_buffer("slopes", sops.distance_slopes(s.heads).to(device) if s.distance_bias else None, persistent=False)
        if s.sink:
            self.sinks = nn.Parameter(torch.zeros(s.heads, **f32))
        else:
            self.register_buffer("sinks", torch.zeros(s.heads, **f32) if s.sink_one else None, persistent=False)
        self.rel = nn.Parameter(torch.zeros(s.bias_rows, s.heads, **f32)) if s.bias_rows else None
        self._table: Optional[torch.Tensor] = None          # the learned bias by distance, formed on first use

    def bias_table(self) -> Optional[torch.Tensor]:
        if self.rel is not None and (self._table is None or self._table.device != self.rel.device):
            self._table = sops.bucket_bias_table(self.rel.detach(), self.spec.bias_max).to(self.rel.device)
        return self._table

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: q, k, v (+ ``.b`` biases), q.norm, k.norm, sink, g, rel ([rows, heads]), o (+ ``o.b``)."""
        s = self.spec
        with torch.no_grad():
            parts = [get(prefix + "q"), get(prefix + "k"), get(prefix + "v")] + ([get(prefix + "g")] if s.out_gate else [])
            self.w_in.copy_(torch.cat(parts, dim=0))
            self.w_o.copy_(get(prefix + "o"))
            if s.bias:
                self.b_in.copy_(torch.cat([get(prefix + "q.b"), get(prefix + "k.b"), get(prefix + "v.b")], dim=0).float())
            if self.b_o is not None:
                self.b_o.copy_(get(prefix + "o.b").float())
            if s.proj_norm:
                self.q_norm.copy_(get(prefix + "q.norm").float())
                self.k_norm.copy_(get(prefix + "k.norm").float())
            if s.sink:
                self.sinks.copy_(get(prefix + "sink").float())
            if self.rel is not None:
                self.rel.copy_(get(prefix + "rel").float())
        self._table = None

    def cache_shape(self, num_blocks: int, block_size: int) -> Tuple[int, ...]:
        return (num_blocks, block_size, self.spec.cache_width)

    def forward(self, h: torch.Tensor, batch, cache: torch.Tensor) -> torch.Tensor:
        """h: [T, W] in the activation type; ``cache``: this layer's [pages, bs, G (d + e)]."""
        s = self.spec
        p = ops.linear(h, self.w_in)
        if self.rotary_append:
            q = wops.window_qkv_write(p, self.b_in, self.q_norm, self.k_norm, s.heads, s.kv_heads, s.dim, s.vdim, s.rot_dims, self.rot_freq, 1.0,
                                      self.eps, batch.positions, batch.slots, cache, batch.block_size, rot_half=True)
        else:
            q = sops.window_kv_append(p, self.b_in, s.heads, s.kv_heads, s.dim, s.vdim, s.value_norm, self.eps, batch.slots, cache,
                                      qk_norm=s.qk_norm, q_temp=s.q_temp, positions=batch.positions)
        gate = p[:, self.n_qkv:] if s.out_gate else None
        # prompt portions: tiles of 128 tokens on the tensor-core kernel, of 16 on the FMA kernel; decoded tokens: one each
        width = sops.tile_width(cache.dtype, s.heads, s.kv_heads, s.dim, s.vdim, q.is_cuda, batch.decode_only)
        o = sops.softcap_window_attention(q, cache, batch.block_tables, batch.tiles(width), 1 if batch.decode_only else width,
                                          batch.positions, gate, self.slopes, self.sinks, s.scale, s.softcap, s.window, s.keep_first,
                                          s.heads, s.kv_heads, s.dim, s.vdim, batch.block_size, h.dtype, max_context=batch.max_context,
                                          table=self.bias_table(), chunk=s.chunk)
        y = ops.linear(o, self.w_o)
        return y if self.b_o is None else torch.add(y, self.b_o)        # fp32 sum: the residual update takes either type


@dataclass
class DifferentialAttentionSpec:
    heads: int
    kv_heads: int
    dim: int            # size of each of the two query / key vectors of a head
    vdim: int           # value size per head
    scale: float
    diff: float         # the constant in lam; the output is multiplied by 1 - diff
    rot_dims: int = 0   # rotated numbers per query / key vector (even, <= dim); 0: no rotation
    rot_base: float = 10000.0
    rot_scaling: Optional[Dict[str, Any]] = None
    head_gate: bool = True      # sigmoid gate per (token, head) from a projection of the mixer's input

    @property
    def cache_width(self) -> int:
        return self.kv_heads * (2 * self.dim + self.vdim)


class DifferentialAttention(nn.Module):
    TILE_TOKENS = dops.TILE_TOKENS      # tile width of the ragged batch this mixer asks for (serve/ragged.py)
    stateful = False

    def __init__(self, width: int, spec: DifferentialAttentionSpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        if s.heads % s.kv_heads or s.rot_dims % 2 or s.rot_dims > s.dim:
            raise ValueError(f"inconsistent attention sizes: {s}")
        self.eps = eps
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        self.nq, self.nk, self.nv = s.heads * 2 * s.dim, s.kv_heads * 2 * s.dim, s.kv_heads * s.vdim
        self.w_in = nn.Parameter(torch.empty(self.nq + self.nk + self.nv + (s.heads if s.head_gate else 0), width, **kw))   # [q ; k ; v ; g]
        self.lam_q = nn.Parameter(torch.zeros(2, s.dim, **f32))
        self.lam_k = nn.Parameter(torch.zeros(2, s.dim, **f32))
        self.w_o = nn.Parameter(torch.empty(width, s.heads * s.vdim, **kw))
        if s.rot_dims:
            f, self.rot_mult = rope_frequencies(s.rot_dims, s.rot_base, s.rot_scaling)
        else:
            f, self.rot_mult = torch.zeros(1), 1.0
        self.register_buffer("rot_freq", f.to(device), persistent=False)
        self._lam: Optional[float] = None

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: q, k, v, g ([heads, width]), lq1, lk1, lq2, lk2, o."""
        s = self.spec
        with torch.no_grad():
            parts = [get(prefix + "q"), get(prefix + "k"), get(prefix + "v")] + ([get(prefix + "g")] if s.head_gate else [])
            self.w_in.copy_(torch.cat(parts, dim=0))
            self.lam_q.copy_(torch.stack([get(prefix + "lq1").float(), get(prefix + "lq2").float()]))
            self.lam_k.copy_(torch.stack([get(prefix + "lk1").float(), get(prefix + "lk2").float()]))
            self.w_o.copy_(get(prefix + "o"))
        self._lam = None

    @property
    def lam(self) -> float:
        """``exp(lq1 . lk1) - exp(lq2 . lk2) + diff``, evaluated once in fp32."""
        if self._lam is None:
            dots = (self.lam_q.detach().float() * self.lam_k.detach().float()).sum(-1).cpu()
            e = torch.exp(dots)
            self._lam = float(e[0] - e[1] + torch.tensor(self.spec.diff, dtype=torch.float32))
        return self._lam

    def cache_shape(self, num_blocks: int, block_size: int) -> Tuple[int, ...]:
        return (num_blocks, block_size, self.spec.cache_width)

    def forward(self, h: torch.Tensor, batch, cache: torch.Tensor) -> torch.Tensor:
        """h: [T, W] in the activation type; ``cache``: this layer run's [pages, bs, G (2 d + e)]."""
        s = self.spec
        p = ops.linear(h, self.w_in)
        q = dops.rotary_kv_append(p, 2 * s.heads, 2 * s.kv_heads, s.dim, self.nv, s.rot_dims, self.rot_freq, self.rot_mult,
                                  batch.positions, batch.slots, cache)
        gate = p[:, self.nq + self.nk + self.nv:] if s.head_gate else None
        # prompt portions: tiles of 128 tokens on the tensor-core kernel, of 16 on the FMA kernel; decoded tokens: one each
        width = dops.tile_width(cache.dtype, s.heads, s.kv_heads, s.dim, s.vdim, q.is_cuda, batch.decode_only)
        o = dops.diff_attention(q, cache, batch.block_tables, batch.tiles(width), 1 if batch.decode_only else width,
                                batch.positions, gate, s.scale, self.lam, 1.0 - s.diff, self.eps, s.heads, s.kv_heads, s.dim, s.vdim,
                                batch.block_size, h.dtype, max_context=batch.max_context)
        return ops.linear(o, self.w_o)


@dataclass
class GatedLinearAttentionSpec:
    heads: int
    dim: int            # query / key size per head
    vdim: int           # value size per head
    tau: float          # the decay is sigmoid(z)^(1/tau)
    decay_rank: int     # inner size of the low-rank decay projection


class GatedLinearAttention(nn.Module):
    stateful = True

    def __init__(self, width: int, spec: GatedLinearAttentionSpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        self.eps = eps
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        self.nk, self.nv = s.heads * s.dim, s.heads * s.vdim
        self.w_in = nn.Parameter(torch.empty(2 * self.nk + 2 * self.nv + s.decay_rank, width, **kw))     # [q ; k ; v ; g ; a1]
        self.w_a2 = nn.Parameter(torch.empty(self.nk, s.decay_rank, **kw))
        self.b_a2 = nn.Parameter(torch.zeros(self.nk, **f32))
        self.norm = nn.Parameter(torch.ones(s.vdim, **f32))
        self.w_o = nn.Parameter(torch.empty(width, self.nv, **kw))

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: q, k, v, g, a1, a2 (+ ``a2.b``), norm, o."""
        with torch.no_grad():
            self.w_in.copy_(torch.cat([get(prefix + n) for n in ("q", "k", "v", "g", "a1")], dim=0))
            self.w_a2.copy_(get(prefix + "a2"))
            self.b_a2.copy_(get(prefix + "a2.b").float())
            self.norm.copy_(get(prefix + "norm").float())
            self.w_o.copy_(get(prefix + "o"))

    def state_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        s = self.spec
        return ((s.heads, s.dim, s.vdim),)

    def forward(self, h: torch.Tensor, batch, state) -> torch.Tensor:
        """h: [T, W] in the activation type; ``state``: (this layer run's [slots, H, d, e] fp32,)."""
        s = self.spec
        nk, nv = self.nk, self.nv
        p = ops.linear(h, self.w_in)
        z = ops.linear(p[:, 2 * nk + 2 * nv:], self.w_a2)
        o = rops.gla_scan(p[:, :nk], p[:, nk:2 * nk], p[:, 2 * nk:2 * nk + nv], z, self.b_a2, batch.portions, state[0], s.heads, s.dim,
                          s.vdim, s.dim ** -0.5, s.tau)
        y = rops.gla_output(o, self.norm, p[:, 2 * nk + nv:2 * nk + 2 * nv], s.heads, s.vdim, self.eps, h.dtype)
        return ops.linear(y, self.w_o)


@dataclass
class SelectiveScanSpec:
    inner: int          # channels
    state: int          # state numbers per channel (N)
    dt_rank: int
    conv: int           # taps of the causal convolution


class SelectiveScan(nn.Module):
    stateful = True

    def __init__(self, width: int, spec: SelectiveScanSpec, dtype, device):
        super().__init__()
        s = self.spec = spec
        if s.conv < 1:
            raise ValueError("the convolution needs at least one tap")
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        self.w_in = nn.Parameter(torch.empty(2 * s.inner, width, **kw))                 # [x ; z]
        self.conv_w = nn.Parameter(torch.empty(s.inner, s.conv, **f32))
        self.conv_b = nn.Parameter(torch.zeros(s.inner, **f32))
        self.w_x = nn.Parameter(torch.empty(s.dt_rank + 2 * s.state, s.inner, **kw))    # [dt ; B ; C]
        self.w_dt = nn.Parameter(torch.empty(s.inner, s.dt_rank, **kw))
        self.dt_bias = nn.Parameter(torch.zeros(s.inner, **f32))
        self.A = nn.Parameter(-torch.ones(s.inner, s.state, **f32))                    # -exp(A_log), fp32
        self.D = nn.Parameter(torch.ones(s.inner, **f32))
        self.w_o = nn.Parameter(torch.empty(width, s.inner, **kw))

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: in, conv (+ ``conv.b``), x, dt (+ ``dt.b``), A_log, D, o."""
        with torch.no_grad():
            self.w_in.copy_(get(prefix + "in"))
            self.conv_w.copy_(get(prefix + "conv").float())
            self.conv_b.copy_(get(prefix + "conv.b").float())
            self.w_x.copy_(get(prefix + "x"))
            self.w_dt.copy_(get(prefix + "dt"))
            self.dt_bias.copy_(get(prefix + "dt.b").float())
            self.A.copy_(-torch.exp(get(prefix + "A_log").float()))
            self.D.copy_(get(prefix + "D").float())
            self.w_o.copy_(get(prefix + "o"))

    def state_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        s = self.spec
        return ((s.inner, s.state), (max(s.conv - 1, 0), s.inner))

    def forward(self, h: torch.Tensor, batch, state) -> torch.Tensor:
        """h: [T, W] in the activation type; ``state``: this layer run's ([slots, C, N], [slots, taps - 1, C]) fp32."""
        s = self.spec
        C, R, N = s.inner, s.dt_rank, s.state
        xz = ops.linear(h, self.w_in)
        x, z = xz[:, :C], xz[:, C:]
        u = rops.causal_conv_silu(x, self.conv_w, self.conv_b, batch.portions, batch.seq_rows, state[1])
        bc = ops.linear(u, self.w_x)
        dtp = ops.linear(bc[:, :R], self.w_dt)
        y = rops.selective_scan(u, bc, R, R + N, dtp, self.dt_bias, self.A, self.D, z, x, batch.portions, state[0], state[1])
        return ops.linear(y, self.w_o)


@dataclass
class DeltaRuleSpec:
    heads: int
    kv_heads: int       # query / key heads: head h reads h // (heads // kv_heads)
    dim: int            # query / key size per head
    vdim: int           # value size per head
    conv: int           # taps of the causal convolutions
    per_channel: bool   # one decay per head and key row from a low-rank projection; otherwise one per head
    decay_rank: int = 0     # inner size of the low-rank decay projection (per_channel)
    gate_rank: int = 0      # inner size of a low-rank output gate; 0: full projection
    gate_act: str = "silu"  # activation of the output gate: silu or sigmoid


class DeltaRule(nn.Module):
    stateful = True

    def __init__(self, width: int, spec: DeltaRuleSpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        if s.heads % s.kv_heads or s.conv < 1 or s.dim > mops.MAX_DIM or (s.per_channel and s.decay_rank < 1):
            raise ValueError(f"inconsistent delta-rule sizes: {s}")
        self.eps = eps
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        H, nk, nv = s.heads, s.kv_heads * s.dim, s.heads * s.vdim
        self.n_qkv = 2 * nk + nv
        # rows of the packed projection: q, k, v without gaps (one convolution runs over them), then parts that start at
        # multiples of 8 (a GEMM reads the latents in place)
        parts = [("a1", s.decay_rank) if s.per_channel else ("a", H), ("g1", s.gate_rank) if s.gate_rank else ("g", nv), ("b", H)]
        self.at: Dict[str, int] = {}
        rows = _pad8(self.n_qkv)
        for name, n in parts:
            self.at[name] = rows
            rows += _pad8(n)
        self.w_in = nn.Parameter(torch.zeros(rows, width, **kw))
        self.conv_w = nn.Parameter(torch.zeros(self.n_qkv, s.conv, **f32))
        self.n_z = H * s.dim if s.per_channel else H
        # low-rank second stages as one block-diagonal matrix over the neighbouring latents [a1 | g1]
        self.low_rows = (self.n_z if s.per_channel else 0) + (nv if s.gate_rank else 0)
        self.low_k = (_pad8(s.decay_rank) if s.per_channel else 0) + _pad8(s.gate_rank)
        self.low_at = self.at["a1"] if s.per_channel else self.at.get("g1", 0)
        self.w_low = nn.Parameter(torch.zeros(_pad8(self.low_rows), self.low_k, **kw)) if self.low_rows else None
        self.dt_bias = nn.Parameter(torch.zeros(self.n_z, **f32))
        self.speed = nn.Parameter(torch.ones(H, **f32))                                     # exp(A_log)
        self.norm = nn.Parameter(torch.ones(s.vdim, **f32))
        self.w_o = nn.Parameter(torch.empty(width, nv, **kw))

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: q, k, v (+ ``.conv``), b, A_log, dt_bias, a1 + a2 or a, g1 + g2 or g, norm, o."""
        s = self.spec
        with torch.no_grad():
            self.w_in.zero_()
            self.w_in[:self.n_qkv].copy_(torch.cat([get(prefix + n) for n in ("q", "k", "v")], dim=0))
            for name, at in self.at.items():
                w = get(prefix + name)
                self.w_in[at:at + w.shape[0]].copy_(w)
            self.conv_w.copy_(torch.cat([get(prefix + n + ".conv").float() for n in ("q", "k", "v")], dim=0))
            if self.w_low is not None:
                self.w_low.zero_()
                r = k = 0
                if s.per_channel:
                    self.w_low[:self.n_z, :s.decay_rank].copy_(get(prefix + "a2"))
                    r, k = self.n_z, _pad8(s.decay_rank)
                if s.gate_rank:
                    self.w_low[r:r + s.heads * s.vdim, k:k + s.gate_rank].copy_(get(prefix + "g2"))
            self.dt_bias.copy_(get(prefix + "dt_bias").float())
            self.speed.copy_(torch.exp(get(prefix + "A_log").float()))
            self.norm.copy_(get(prefix + "norm").float())
            self.w_o.copy_(get(prefix + "o"))

    def state_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        s = self.spec
        return ((s.heads, s.dim, s.vdim), (s.conv - 1, self.n_qkv))

    def forward(self, h: torch.Tensor, batch, state) -> torch.Tensor:
        """h: [T, W] in the activation type; ``state``: this layer run's ([slots, H, d, e], [slots, taps - 1, C]) fp32."""
        s = self.spec
        p = ops.linear(h, self.w_in)
        low = ops.linear(p[:, self.low_at:self.low_at + self.low_k], self.w_low) if self.w_low is not None else None
        nv = s.heads * s.vdim
        z = low[:, :self.n_z] if s.per_channel else p[:, self.at["a"]:self.at["a"] + s.heads]
        if s.gate_rank:
            at = self.n_z if s.per_channel else 0
            gate = low[:, at:at + nv]
        else:
            gate = p[:, self.at["g"]:self.at["g"] + nv]
        y = mops.delta_rule(p[:, :self.n_qkv], self.conv_w, z, self.dt_bias, self.speed, p[:, self.at["b"]:self.at["b"] + s.heads], gate,
                            self.norm, batch.portions, batch.seq_rows, state[0], state[1], s.heads, s.kv_heads, s.dim, s.vdim,
                            s.per_channel, self.eps, s.gate_act, decode=batch.decode_only)
        return ops.linear(y, self.w_o)


@dataclass
class BonusMemorySpec:
    heads: int
    dim: int            # key and value size per head
    decay_rank: int     # inner size of the low-rank decay projection


class BonusMemory(nn.Module):
    stateful = True
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, width: int, spec: BonusMemorySpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        if s.dim > mops.MAX_DIM or s.decay_rank < 1:
            raise ValueError(f"inconsistent time-mixing sizes: {s}")
        self.eps = eps
        kw = dict(dtype=dtype, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        n = s.heads * s.dim
        self.mu = nn.Parameter(torch.zeros(len(self.MIXES), width, **f32))
        self.w_rkvg = nn.Parameter(torch.empty(4, n, width, **kw))
        self.w_1 = nn.Parameter(torch.zeros(_pad8(s.decay_rank), width, **kw))
        self.w_2 = nn.Parameter(torch.zeros(n, _pad8(s.decay_rank), **kw))
        self.w_0 = nn.Parameter(torch.zeros(n, **f32))
        self.u = nn.Parameter(torch.zeros(n, **f32))
        self.norm = nn.Parameter(torch.ones(n, **f32))
        self.w_o = nn.Parameter(torch.empty(width, n, **kw))

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: mu.{r,k,v,g,w}, r, k, v, g, w1, w2, w0, u ([heads, dim]), norm, o."""
        r = self.spec.decay_rank
        with torch.no_grad():
            for i, name in enumerate(self.MIXES):
                self.mu[i].copy_(get(prefix + "mu." + name).float())
            for i, name in enumerate(self.MIXES[:4]):
                self.w_rkvg[i].copy_(get(prefix + name))
            self.w_1.zero_()
            self.w_2.zero_()
            self.w_1[:r].copy_(get(prefix + "w1"))
            self.w_2[:, :r].copy_(get(prefix + "w2"))
            self.w_0.copy_(get(prefix + "w0").float())
            self.u.copy_(get(prefix + "u").float().reshape(-1))
            self.norm.copy_(get(prefix + "norm").float())
            self.w_o.copy_(get(prefix + "o"))

    def state_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        s = self.spec
        return ((s.heads, s.dim, s.dim), (self.mu.shape[1],))

    def forward(self, h: torch.Tensor, batch, state) -> torch.Tensor:
        """h: [T, W] in the activation type; ``state``: this layer run's ([slots, H, d, d], [slots, W]) fp32."""
        s = self.spec
        mix = mops.token_shift(h, self.mu, batch.portions, batch.seq_rows, state[1])
        r, k, v, g = torch.bmm(mix[:4], self.w_rkvg.transpose(1, 2)).unbind(0)
        z = ops.linear(tanh_(ops.linear(mix[4], self.w_1)), self.w_2)
        y = mops.bonus_memory(r, k, v, z, self.w_0, self.u, g, self.norm, h, batch.portions, state[0], state[1], s.heads, s.dim, self.eps,
                              decode=batch.decode_only)
        return ops.linear(y, self.w_o)


@dataclass
class RetentionSpec:
    heads: int
    dim: int            # query / key size per head
    vdim: int           # value size per head
    decay: Tuple[float, ...]    # one per head
    rot_dims: int = 0   # rotated numbers per head, pairs (i, i + rot_dims/2); 0: no rotation
    rot_base: float = 10000.0


class Retention(nn.Module):
    stateful = True

    def __init__(self, width: int, spec: RetentionSpec, eps: float, dtype, device):
        super().__init__()
        s = self.spec = spec
        if len(s.decay) != s.heads or s.dim > retops.MAX_DIM or s.rot_dims % 2 or s.rot_dims > s.dim:
            raise ValueError(f"inconsistent retention sizes: {s}")
        self.eps = eps
        nk, nv = s.heads * s.dim, s.heads * s.vdim
        self.at: Dict[str, Tuple[int, int]] = {}         # columns of the packed projection, parts starting at multiples of 8
        rows = 0
        for name, n in (("q", nk), ("k", nk), ("v", nv), ("g", nv)):
            self.at[name] = (rows, rows + n)
            rows += _pad8(n)
        self.w_in = nn.Parameter(torch.zeros(rows, width, dtype=dtype, device=device))
        self.w_o = nn.Parameter(torch.empty(width, nv, dtype=dtype, device=device))
        freq = rope_frequencies(s.rot_dims, s.rot_base)[0] if s.rot_dims else torch.zeros(1)
        self.register_buffer("rot_freq", freq.to(device), persistent=False)
        decay_m1 = torch.tensor([float(g) - 1.0 for g in s.decay], dtype=torch.float64).to(torch.float32)
        self.register_buffer("decay_m1", decay_m1.to(device), persistent=False)

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: q, k, v, g, o."""
        with torch.no_grad():
            self.w_in.zero_()
            for name, (a, b) in self.at.items():
                self.w_in[a:b].copy_(get(prefix + name))
            self.w_o.copy_(get(prefix + "o"))

    def state_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        s = self.spec
        return ((s.heads, s.dim, s.vdim),)

    def forward(self, h: torch.Tensor, batch, state) -> torch.Tensor:
        """h: [T, W] in the activation type; ``state``: (this layer run's [slots, H, d, e] fp32,)."""
        s = self.spec
        p = ops.linear(h, self.w_in)
        q, k, v, g = (p[:, a:b] for a, b in self.at.values())
        y = retops.retention(q, k, v, g, batch.positions, self.rot_freq, s.rot_dims, self.decay_m1, batch.portions, state[0], s.heads, s.dim,
                             s.vdim, self.eps, decode=batch.decode_only, tiles=batch.tiles(retops.CHUNK))
        return ops.linear(y, self.w_o)


class BranchPair(nn.Module):
    def __init__(self, width: int, left: nn.Module, right: nn.Module, device):
        super().__init__()
        self.left, self.right = left, right
        f32 = dict(dtype=torch.float32, device=device)
        self.left_w = nn.Parameter(torch.ones(width, **f32))
        self.right_w = nn.Parameter(torch.ones(width, **f32))

    def load(self, get, prefix: str) -> None:
        """Checkpoint names under ``prefix``: left.*, right.* (the branches'), left.out, right.out."""
        self.left.load(get, prefix + "left.")
        self.right.load(get, prefix + "right.")
        with torch.no_grad():
            self.left_w.copy_(get(prefix + "left.out").float())
            self.right_w.copy_(get(prefix + "right.out").float())

    def forward(self, h: torch.Tensor, batch, own) -> BranchSum:
        """``own``: (the left branch's cache or states, the right branch's)."""
        return BranchSum(self.left(h, batch, own[0]), self.right(h, batch, own[1]), self.left_w, self.right_w, 0.5)
