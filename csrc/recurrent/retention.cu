// Retention as a recurrence over a per-sequence state, for ragged batches (portions of prompts next to single decoded tokens), bf16
// or fp32 projections.  S: [d, e] fp32 per head, zero before a sequence's first token, kept in the sequence's state slot.
//
//       q, k <- rotated by position: pairs (i, i + rot/2) of the first rot numbers turn by position * freq_i;   k <- k / sqrt(d)
//       S <- decay_h S + k v^T;   o = S^T q                                  a fixed decay per head
//
//   llmctl_retention_prepare : fully parallel over tokens: rotated queries and keys, values and q . k in fp32, padded so that the
//       scan copies whole 16-byte rows.
//   llmctl_retention_scan : the serial part (the matrix-state scan, kind 3; any sizes).
//   llmctl_retention_step : one decoded token per sequence in ONE launch: rotation, state update, read-out, the head's RMS norm
//       and output gate.
//   llmctl_retention_chunked : prompts in bf16 (sizes below), chunks of 64 tokens as matrix products on the tensor cores
//       (mma.sync m16n8k16) instead of the serial scan.  With local indices i, j in a chunk of L tokens and S before it:
//           o_i = decay^(i+1) q_i^T S + sum_(j <= i) decay^(i-j) (q_i . k_j) v_j
//           S  <- decay^L S + sum_j decay^(L-1-j) k_j v_j^T
//       Four launches: sines and cosines per (token, pair); the sums over j of every chunk and head (parallel); the chain over the
//       chunks, elementwise in fp32, which leaves the state before every chunk; outputs with the head's RMS norm and gate
//       (parallel).  Rotated queries and keys, decayed scores and states enter the products as bf16 pairs hi + lo (exact to
//       ~2^-17; values are bf16 already), accumulators and the carried state are fp32.
// The decay is applied as S + (decay - 1) S.  Everything is fp32; only the projections and the gated output have the activation type.
// Reference: none (the reference has no model code).
#include "matrix_state.cuh"

namespace llmctl {

struct RetentionPrepParams {
  const void* q;              // [T, H d] (row strides below)
  const void* k;
  const void* v;              // [T, H e]
  long long ldq, ldk, ldv;
  const int* positions;
  const float* freq;          // [rot / 2]
  const float* dm;            // [H] decay minus one
  int H, d, e, rot;
  MsWork w;
};

// Rotated value of coordinate c of a head's numbers x (pairs (c, c + rot/2)); cs: (cos, sin) per pair.
template <typename T>
__device__ __forceinline__ float ms_rotate_half(const T* x, int c, int rot, const float2* cs) {
  const float v = to_f32(x[c]);
  if (c >= rot) return v;
  const int half = rot >> 1;
  const float2 a = cs[c < half ? c : c - half];
  return c < half ? v * a.x - to_f32(x[c + half]) * a.y : v * a.x + to_f32(x[c - half]) * a.y;
}

// One CTA per token, a warp per head in turn; the token's sines and cosines are evaluated once.
template <typename T, int NI>
__global__ void __launch_bounds__(256)
retention_prepare_kernel(const RetentionPrepParams p) {
  __shared__ float2 cs[128];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, H = p.H, d = p.d, e = p.e;
  const int dp = ms_pad_rows(d), ep = ms_pad_cols(e);
  const long long t = blockIdx.x;
  const float pos = static_cast<float>(p.positions[t]);
  for (int i = threadIdx.x; i < p.rot >> 1; i += blockDim.x) {
    float s, c;
    sincosf(pos * p.freq[i], &s, &c);
    cs[i] = make_float2(c, s);
  }
  __syncthreads();
  const float ks = 1.f / sqrtf(static_cast<float>(d));
  for (int h = blockIdx.y * 8 + warp; h < H; h += gridDim.y * 8) {
    const long long row = t * H + h;
    const T* q = static_cast<const T*>(p.q) + t * p.ldq + h * d;
    const T* k = static_cast<const T*>(p.k) + t * p.ldk + h * d;
    const T* v = static_cast<const T*>(p.v) + t * p.ldv + h * e;
    float qk = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = lane + 32 * i;
      float a = 0.f, b = 0.f;
      if (c < d) {
        a = ms_rotate_half(q, c, p.rot, cs);
        b = ms_rotate_half(k, c, p.rot, cs) * ks;
      }
      p.w.q[row * dp + c] = a;
      p.w.k[row * dp + c] = b;
      qk += a * b;
    }
    for (int c = lane; c < ep; c += 32) p.w.v[row * ep + c] = c < e ? to_f32(v[c]) : 0.f;
    qk = warp_sum(qk);
    if (lane == 0) *reinterpret_cast<float4*>(p.w.sc + row * 4) = make_float4(1.f, qk, p.dm[h], 0.f);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// chunks of 64 tokens on the tensor cores
// ---------------------------------------------------------------------------------------------------------------
constexpr int kRcTokens = 64;
constexpr int kRcEarly = 2;         // stages of 16 state rows that the output kernel fills before it has read the keys
constexpr int kRcFlight = 6;        // most slices of the state in flight

struct RetentionChunkParams {
  const __nv_bfloat16* q;     // [T, H d] (row strides below)
  const __nv_bfloat16* k;
  const __nv_bfloat16* v;     // [T, H e]
  const __nv_bfloat16* gate;  // [T, H e]
  long long ldq, ldk, ldv, ldg;
  const float2* cs;           // [T, half] (cos, sin)
  int half;                   // rotated pairs per head
  const float* dm;            // [H] decay minus one
  const int* portions;
  int nportions;
  const int* tiles;           // [chunks, 4] = (first token row, tokens, portion, 0), portions in order
  float* state;               // [slots, H, d, e]
  float* scratch;             // [chunks, nh, d, e]: a chunk's sum, then groups of 8 numbers of the state before it as 8 hi, 8 lo
  __nv_bfloat16* out;         // [T, H e]
  int H, d, e, h0, nh;        // heads h0 .. h0 + nh - 1
  int gate_sigmoid;
  float eps;
};

__global__ void __launch_bounds__(256)
retention_angles_kernel(const int* __restrict__ positions, const float* __restrict__ freq, int half, float2* __restrict__ cs, int tokens) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= tokens * half) return;
  float s, c;
  sincosf(static_cast<float>(positions[i / half]) * freq[i % half], &s, &c);
  cs[i] = make_float2(c, s);
}

__device__ __forceinline__ float rc_log2_decay(float dm) { return log1pf(dm) * 1.4426950408889634f; }
__device__ __forceinline__ float rc_power(float log2_decay, int n) { return n == 0 ? 1.f : exp2f(log2_decay * static_cast<float>(n)); }

// four fp32 numbers as bf16 pairs hi + lo
__device__ __forceinline__ void rc_split4(const float (&v)[4], uint2& hi, uint2& lo) {
  float r[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) r[i] = v[i] - __bfloat162float(__float2bfloat16(v[i]));
  hi = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  lo = make_uint2(pack_bf16x2(r[0], r[1]), pack_bf16x2(r[2], r[3]));
}

// Rows j of a chunk (x[m] + j ld[m], d numbers each, NM operands): rotated, times factor[m] [* decay^(last - j)], split into hi and lo
// [64][d + 8] in shared memory; rows past n are zeros.  An item is four pairs or four unrotated numbers of every operand; the
// loads of IT items per thread are in flight together.
template <int NM, int IT, bool DECAY>
__device__ __forceinline__ void rc_load_rotated(const __nv_bfloat16* const (&x)[NM], const long long (&ld)[NM], const float2* cs, int half, int d, int n,
                                                const float (&factor)[NM], float log2_decay, int last, __nv_bfloat16* const (&hi)[NM],
                                                __nv_bfloat16* const (&lo)[NM]) {
  const int pairs = half >> 2, per = (d >> 2) - pairs, lds = d + 8, total = kRcTokens * per;
  const int dj = 256 / per, dk = 256 - dj * per;       // CTAs of 256 threads
  int i = threadIdx.x, j = i / per, k = i - j * per;
  while (i < total) {
    uint2 a[IT][NM], b[IT][NM];
    float w[IT][8];
    int jj[IT], cc[IT];
#pragma unroll
    for (int u = 0; u < IT; ++u) {
      jj[u] = i < total ? j : -1;
      cc[u] = k < pairs ? k << 2 : (k << 2) + half;
#pragma unroll
      for (int m = 0; m < NM; ++m) a[u][m] = b[u][m] = make_uint2(0u, 0u);
      if (i < total && j < n) {
#pragma unroll
        for (int m = 0; m < NM; ++m) a[u][m] = *reinterpret_cast<const uint2*>(x[m] + j * ld[m] + cc[u]);
        if (cc[u] < half) {
#pragma unroll
          for (int m = 0; m < NM; ++m) b[u][m] = *reinterpret_cast<const uint2*>(x[m] + j * ld[m] + cc[u] + half);
          const float* t = reinterpret_cast<const float*>(cs + j * half + cc[u]);
          *reinterpret_cast<float4*>(w[u]) = *reinterpret_cast<const float4*>(t);
          *reinterpret_cast<float4*>(w[u] + 4) = *reinterpret_cast<const float4*>(t + 4);
        }
      }
      i += 256;
      j += dj;
      k += dk;
      if (k >= per) k -= per, ++j;
    }
#pragma unroll
    for (int u = 0; u < IT; ++u) {
      const int row = jj[u], c = cc[u];
      if (row < 0) continue;
      float pw = 1.f;
      if (DECAY) pw = row < n ? rc_power(log2_decay, last - row) : 0.f;
      const int at = row * lds + c;
#pragma unroll
      for (int m = 0; m < NM; ++m) {
        const float f = factor[m] * pw;
        float p[4] = {__uint_as_float(a[u][m].x << 16), __uint_as_float(a[u][m].x & 0xffff0000u), __uint_as_float(a[u][m].y << 16),
                      __uint_as_float(a[u][m].y & 0xffff0000u)};
        uint2 h, l;
        if (c < half) {
          float q[4] = {__uint_as_float(b[u][m].x << 16), __uint_as_float(b[u][m].x & 0xffff0000u), __uint_as_float(b[u][m].y << 16),
                        __uint_as_float(b[u][m].y & 0xffff0000u)};
          if (row < n) {
#pragma unroll
            for (int v = 0; v < 4; ++v) {
              const float p0 = p[v], q0 = q[v];
              p[v] = (p0 * w[u][2 * v] - q0 * w[u][2 * v + 1]) * f;
              q[v] = (q0 * w[u][2 * v] + p0 * w[u][2 * v + 1]) * f;
            }
          }
          rc_split4(q, h, l);
          *reinterpret_cast<uint2*>(hi[m] + at + half) = h;
          *reinterpret_cast<uint2*>(lo[m] + at + half) = l;
        } else {
#pragma unroll
          for (int v = 0; v < 4; ++v) p[v] *= f;
        }
        rc_split4(p, h, l);
        *reinterpret_cast<uint2*>(hi[m] + at) = h;
        *reinterpret_cast<uint2*>(lo[m] + at) = l;
      }
    }
  }
}

// asynchronous copies of a chunk's rows (rows past n: zeros); the caller commits and waits
__device__ __forceinline__ void rc_load_rows(const __nv_bfloat16* x, long long ld, int cols, int n, __nv_bfloat16* dst, int lds) {
  const int per = cols >> 3, dj = 256 / per, dk = 256 - dj * per;
  int j = threadIdx.x / per, k = threadIdx.x - j * per;
  for (; j < kRcTokens; j += dj, k += dk) {
    if (k >= per) {
      k -= per;
      if (++j >= kRcTokens) break;
    }
    const int c = k << 3;
    if (j < n) cp_async_16(dst + j * lds + c, x + j * ld + c);
    else *reinterpret_cast<uint4*>(dst + j * lds + c) = make_uint4(0u, 0u, 0u, 0u);
  }
}

// A fragment of A[m][k] = s[k0 + k][m0 + m] (operand stored [k][m] row-major): ldmatrix with transposition
__device__ __forceinline__ void rc_a_frag_km(uint32_t (&a)[4], const __nv_bfloat16* s, int ld, int m0, int k0, int lane) {
  const __nv_bfloat16* p = s + (k0 + (lane & 7) + ((lane >> 4) << 3)) * ld + m0 + (((lane >> 3) & 1) << 3);
  const uint32_t addr = static_cast<uint32_t>(__cvta_generic_to_shared(p));
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3])
               : "r"(addr));
}

// scratch[chunk, head] = sum_j decay^(L-1-j) k_j v_j^T.  Grid: (chunks, heads); a warp owns blocks of 16 x 32 numbers.
__global__ void __launch_bounds__(256, 3)
retention_chunk_sum_kernel(const RetentionChunkParams p) {
  extern __shared__ __align__(16) unsigned char rc_smem[];
  const int d = p.d, e = p.e, ldk = d + 8, ldv = e + 8, h = p.h0 + blockIdx.y;
  const int* tile = p.tiles + 4 * blockIdx.x;
  const long long t0 = tile[0];
  const int n = tile[1];
  if (n <= 0) return;
  __nv_bfloat16* Kh = reinterpret_cast<__nv_bfloat16*>(rc_smem);
  __nv_bfloat16* Kl = Kh + kRcTokens * ldk;
  __nv_bfloat16* V = Kl + kRcTokens * ldk;
  const float lg = rc_log2_decay(p.dm[h]);
  rc_load_rows(p.v + t0 * p.ldv + h * e, p.ldv, e, n, V, ldv);
  cp_async_commit();
  rc_load_rotated<1, 4, true>({p.k + t0 * p.ldk + h * d}, {p.ldk}, p.cs + t0 * p.half, p.half, d, n, {1.f / sqrtf(static_cast<float>(d))}, lg, n - 1,
                              {Kh}, {Kl});
  cp_async_wait_all();
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int nb = (e + 31) / 32, blocks = (d / 16) * nb, steps = (n + 15) / 16;
  float* dst = p.scratch + (static_cast<long long>(blockIdx.x) * p.nh + blockIdx.y) * d * e;
  for (int b = warp; b < blocks; b += 8) {
    const int m0 = b / nb * 16, n0 = b % nb * 32;
    float acc[4][4] = {};
    for (int ks = 0; ks < steps; ++ks) {
      uint32_t ah[4], al[4];
      rc_a_frag_km(ah, Kh, ldk, m0, ks * 16, lane);
      rc_a_frag_km(al, Kl, ldk, m0, ks * 16, lane);
#pragma unroll
      for (int i = 0; i < 4; i += 2)
        if (n0 + 8 * i < e) {                          // e is a multiple of 16
          uint32_t bf[4];
          load_b2_frag_kn(bf, V, ldv, ks * 16, n0 + 8 * i, lane);
          mma_bf16_16816(acc[i], ah, bf[0], bf[1]);
          mma_bf16_16816(acc[i + 1], ah, bf[2], bf[3]);
          mma_bf16_16816(acc[i], al, bf[0], bf[1]);
          mma_bf16_16816(acc[i + 1], al, bf[2], bf[3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (n0 + 8 * i < e) {
        float* o = dst + static_cast<long long>(m0 + g) * e + n0 + 8 * i + 2 * t;
        *reinterpret_cast<float2*>(o) = make_float2(acc[i][0], acc[i][1]);
        *reinterpret_cast<float2*>(o + 8 * e) = make_float2(acc[i][2], acc[i][3]);
      }
  }
}

// The chain over a portion's chunks, eight numbers of a head's state per thread.  Grid: (portions, heads, d e / 2048).
__global__ void __launch_bounds__(256)
retention_chunk_chain_kernel(const RetentionChunkParams p) {
  constexpr int AHEAD = 4;
  const int* pt = p.portions + 4 * blockIdx.x;
  const int n = pt[1], slot = pt[3], h = p.h0 + blockIdx.y;
  const long long numbers = static_cast<long long>(p.d) * p.e, i = (static_cast<long long>(blockIdx.z) * blockDim.x + threadIdx.x) * 8;
  if (n <= 0 || i >= numbers) return;
  int first = 0;
  for (int b = 0; b < static_cast<int>(blockIdx.x); ++b) first += (max(p.portions[4 * b + 1], 0) + kRcTokens - 1) / kRcTokens;
  const int chunks = (n + kRcTokens - 1) / kRcTokens;
  float* st = slot >= 0 ? p.state + (static_cast<long long>(slot) * p.H + h) * numbers + i : nullptr;
  float S[8];
#pragma unroll
  for (int k = 0; k < 8; ++k) S[k] = 0.f;
  if (st && pt[2] > 0) load8_f32(st, S);
  const float lg = log1pf(p.dm[h]);
  const float full = expm1f(lg * kRcTokens), rest = expm1f(lg * static_cast<float>(n - (chunks - 1) * kRcTokens));
  const long long step = static_cast<long long>(p.nh) * numbers;
  float* x = p.scratch + (static_cast<long long>(first) * p.nh + blockIdx.y) * numbers + i;
  float kv[AHEAD][8];
#pragma unroll
  for (int a = 0; a < AHEAD; ++a)
    if (a < chunks) load8_f32(x + a * step, kv[a]);
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      const int c = c0 + a;
      if (c >= chunks) break;
      float r[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) r[k] = S[k] - __bfloat162float(__float2bfloat16(S[k]));
      __nv_bfloat16* pair = reinterpret_cast<__nv_bfloat16*>(x + c * step);       // in place: 8 hi, 8 lo
      store8_f32(pair, S);
      store8_f32(pair + 8, r);
      const float gm = c + 1 < chunks ? full : rest;
#pragma unroll
      for (int k = 0; k < 8; ++k) S[k] = fmaf(gm, S[k], S[k]) + kv[a][k];
      if (c + AHEAD < chunks) load8_f32(x + (c + AHEAD) * step, kv[a]);
    }
  }
  if (st) store8_f32(st, S);
}

// Outputs of a chunk and head (FULL: e == 16 NT).  Warp (r, c) = (warp % 4, warp / 4) owns 16 tokens and half of the value columns (NT tiles of 8).
template <int NT, bool FULL>
__global__ void __launch_bounds__(256, NT <= 8 ? 2 : 1)
retention_chunk_output_kernel(const RetentionChunkParams p) {
  extern __shared__ __align__(16) unsigned char rc_smem[];
  __shared__ float row_ss[2][kRcTokens], power[kRcTokens + 1];      // power[i] = decay^i
  const int d = p.d, e = p.e, ldq = d + 8, ldv = e + 8, h = p.h0 + blockIdx.y;
  const int* tile = p.tiles + 4 * blockIdx.x;
  const long long t0 = tile[0];
  const int n = tile[1];
  if (n <= 0) return;
  const int* pt = p.portions + 4 * tile[2];
  const bool has_state = t0 > pt[0] || (pt[2] > 0 && pt[3] >= 0);      // the first chunk of a sequence starts from zeros
  __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(rc_smem);
  __nv_bfloat16* Ql = Qh + kRcTokens * ldq;
  __nv_bfloat16* V = Ql + kRcTokens * ldq;
  __nv_bfloat16* ring = V + kRcTokens * ldv;           // stages of 16 state rows (hi, lo): kRcEarly of them for their own ...
  __nv_bfloat16* Kh = ring + kRcEarly * 32 * ldv;      // ... and the keys' place, which holds as many more afterwards as fit
  __nv_bfloat16* Kl = Kh + kRcTokens * ldq;
  const float2* cs = p.cs + t0 * p.half;
  const float lg = rc_log2_decay(p.dm[h]);
  const int slices = has_state ? d / 16 : 0, stages = kRcEarly + 128 * ldq / (32 * ldv);
  const int per = e >> 3, dr = 256 / per, dk = 256 - dr * per, first_r = threadIdx.x / per, first_k = threadIdx.x - first_r * per;
  const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.scratch + (static_cast<long long>(blockIdx.x) * p.nh + blockIdx.y) * d * e);
  auto fetch = [&](int sl) {                           // rows 16 sl .. of the state; 8 hi and 8 lo numbers lie next to each other
    __nv_bfloat16* Sh = ring + (sl % stages) * 32 * ldv;
    for (int r = first_r, k = first_k; r < 16; r += dr, k += dk) {
      if (k >= per) {
        k -= per;
        if (++r >= 16) break;
      }
      const int c = k << 3;
      const __nv_bfloat16* u = src + ((sl * 16 + r) * e + c) * 2;
      cp_async_16(Sh + r * ldv + c, u);
      cp_async_16(Sh + (16 + r) * ldv + c, u + 8);
    }
  };
  if (threadIdx.x <= kRcTokens) power[threadIdx.x] = rc_power(lg, threadIdx.x);
  rc_load_rows(p.v + t0 * p.ldv + h * e, p.ldv, e, n, V, ldv);
  cp_async_commit();
  for (int sl = 0; sl < kRcEarly; ++sl) {              // one group per slice from here on, empty past the last one
    if (sl < slices) fetch(sl);
    cp_async_commit();
  }
  rc_load_rotated<2, 4, false>({p.q + t0 * p.ldq + h * d, p.k + t0 * p.ldk + h * d}, {p.ldq, p.ldk}, cs, p.half, d, n,
                               {1.f, 1.f / sqrtf(static_cast<float>(d))}, 0.f, 0, {Qh, Kh}, {Ql, Kl});
  __syncthreads();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int rg = warp & 3, r0 = rg * 16, n_base = (warp >> 2) * NT * 8;
  const bool active = r0 < n;
  uint32_t ph[4][4], pl[4][4];                         // decayed scores, A fragments of 16 keys each
  if (active) {
    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
    for (int ks = 0; ks < d; ks += 16) {
      uint32_t ah[4], al[4];
      load_a_frag(ah, Qh, ldq, r0, ks, lane);
      load_a_frag(al, Ql, ldq, r0, ks, lane);
#pragma unroll
      for (int i = 0; i < 8; i += 2)
        if (i < 2 * (rg + 1)) {                        // later keys are masked for all rows of the warp
          uint32_t bh[4], bl[4];
          load_b2_frag_nk(bh, Kh, ldq, 8 * i, ks, lane);
          load_b2_frag_nk(bl, Kl, ldq, 8 * i, ks, lane);
          mma_bf16_16816(s[i], ah, bh[0], bh[1]);
          mma_bf16_16816(s[i + 1], ah, bh[2], bh[3]);
          mma_bf16_16816(s[i], al, bh[0], bh[1]);
          mma_bf16_16816(s[i + 1], al, bh[2], bh[3]);
          mma_bf16_16816(s[i], ah, bl[0], bl[1]);
          mma_bf16_16816(s[i + 1], ah, bl[2], bl[3]);
        }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int dist = r0 + g + (j >> 1) * 8 - (8 * i + 2 * t + (j & 1));
        s[i][j] = dist >= 0 ? s[i][j] * power[dist] : 0.f;
      }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk)
#pragma unroll
      for (int j = 0; j < 4; ++j) {                    // fragment register j: rows g (+8 for odd j), keys 2t, 2t + 1 (+8 for j >= 2)
        const float a = s[2 * kk + (j >> 1)][(j & 1) * 2], b = s[2 * kk + (j >> 1)][(j & 1) * 2 + 1];
        const float ra = a - __bfloat162float(__float2bfloat16(a)), rb = b - __bfloat162float(__float2bfloat16(b));
        ph[kk][j] = pack_bf16x2(a, b);
        pl[kk][j] = pack_bf16x2(ra, rb);
      }
  }
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  if (has_state) {                                     // uniform over the CTA
    __syncthreads();                                   // the readers of the keys are done
    for (int sl = kRcEarly; sl < kRcFlight; ++sl) {    // kRcFlight groups in flight
      if (sl < slices && sl < stages) fetch(sl);
      cp_async_commit();
    }
    const int ahead = min(stages, kRcFlight);          // slices asked for so far
    for (int sl = 0; sl < slices; ++sl) {
      // slice s >= ahead is in group kRcFlight + s + 1 - ahead: at most kRcFlight - 2 younger groups may be pending, none with a short ring
      if (ahead == kRcFlight) asm volatile("cp.async.wait_group %0;\n" ::"n"(kRcFlight - 2) : "memory");
      else cp_async_wait_all();
      __syncthreads();                                 // slice sl has landed, everyone is done with slice sl - 1
      const int next = sl - 1 + ahead;                 // goes where slice sl - 1 (or nothing yet) was
      if (sl > 0 && next < slices) fetch(next);
      cp_async_commit();
      if (active) {
        const __nv_bfloat16* Sh = ring + (sl % stages) * 32 * ldv;
        const __nv_bfloat16* Sl = Sh + 16 * ldv;
        uint32_t ah[4], al[4];
        load_a_frag(ah, Qh, ldq, r0, sl * 16, lane);
        load_a_frag(al, Ql, ldq, r0, sl * 16, lane);
#pragma unroll
        for (int i = 0; i < NT; i += 2)
          if (FULL || n_base + 8 * i < e) {
            uint32_t bh[4], bl[4];
            load_b2_frag_kn(bh, Sh, ldv, 0, n_base + 8 * i, lane);
            load_b2_frag_kn(bl, Sl, ldv, 0, n_base + 8 * i, lane);
            mma_bf16_16816(acc[i], ah, bh[0], bh[1]);
            mma_bf16_16816(acc[i + 1], ah, bh[2], bh[3]);
            mma_bf16_16816(acc[i], al, bh[0], bh[1]);
            mma_bf16_16816(acc[i + 1], al, bh[2], bh[3]);
            mma_bf16_16816(acc[i], ah, bl[0], bl[1]);
            mma_bf16_16816(acc[i + 1], ah, bl[2], bl[3]);
          }
      }
    }
    const float f_lo = power[r0 + g + 1], f_hi = power[r0 + g + 9];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      acc[i][0] *= f_lo, acc[i][1] *= f_lo;
      acc[i][2] *= f_hi, acc[i][3] *= f_hi;
    }
  }
  uint32_t gz[2][NT];                                  // gates, asked for before the last products
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = r0 + g + 8 * half;
    const __nv_bfloat16* gr = p.gate + (t0 + min(r, n - 1)) * p.ldg + h * e + n_base + 2 * t;
#pragma unroll
    for (int i = 0; i < NT; ++i)
      if (FULL || n_base + 8 * i < e) gz[half][i] = *reinterpret_cast<const uint32_t*>(gr + 8 * i);
  }
  if (!has_state) {                                    // the values' copies may still be in flight
    cp_async_wait_all();
    __syncthreads();
  }
  if (active) {
#pragma unroll
    for (int kk = 0; kk < 4; ++kk)
      if (kk <= rg) {
#pragma unroll
        for (int i = 0; i < NT; i += 2)
          if (FULL || n_base + 8 * i < e) {
            uint32_t b[4];
            load_b2_frag_kn(b, V, ldv, kk * 16, n_base + 8 * i, lane);
            mma_bf16_16816(acc[i], ph[kk], b[0], b[1]);
            mma_bf16_16816(acc[i + 1], ph[kk], b[2], b[3]);
            mma_bf16_16816(acc[i], pl[kk], b[0], b[1]);
            mma_bf16_16816(acc[i + 1], pl[kk], b[2], b[3]);
          }
      }
    float s_lo = 0.f, s_hi = 0.f;
#pragma unroll
    for (int i = 0; i < NT; ++i)
      if (n_base + 8 * i < e) {
        s_lo += acc[i][0] * acc[i][0] + acc[i][1] * acc[i][1];
        s_hi += acc[i][2] * acc[i][2] + acc[i][3] * acc[i][3];
      }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      s_lo += __shfl_xor_sync(0xffffffffu, s_lo, o);
      s_hi += __shfl_xor_sync(0xffffffffu, s_hi, o);
    }
    if (t == 0) row_ss[warp >> 2][r0 + g] = s_lo, row_ss[warp >> 2][r0 + g + 8] = s_hi;
  }
  __syncthreads();
  if (!active) return;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = r0 + g + 8 * half;
    if (r >= n) continue;
    const float f = 1.f / sqrtf((row_ss[0][r] + row_ss[1][r]) / static_cast<float>(e) + p.eps);
    const long long tok = t0 + r;
    __nv_bfloat16* o = p.out + (tok * p.H + h) * e;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int c = n_base + 8 * i + 2 * t;
      if (FULL || n_base + 8 * i < e) {
        const float2 z = make_float2(__uint_as_float(gz[half][i] << 16), __uint_as_float(gz[half][i] & 0xffff0000u));
        // bf16 gates carry 8 bits: the hardware's exponential and reciprocal are exact enough
        const float a0 = __fdividef(p.gate_sigmoid ? 1.f : z.x, 1.f + __expf(-fmaxf(z.x, -80.f)));
        const float a1 = __fdividef(p.gate_sigmoid ? 1.f : z.y, 1.f + __expf(-fmaxf(z.y, -80.f)));
        *reinterpret_cast<__nv_bfloat162*>(o + c) = __floats2bfloat162_rn(acc[i][2 * half] * f * a0, acc[i][2 * half + 1] * f * a1);
      }
    }
  }
}

static size_t rc_sum_smem(int d, int e) { return sizeof(__nv_bfloat16) * kRcTokens * (2 * static_cast<size_t>(d + 8) + (e + 8)); }
static size_t rc_output_smem(int d, int e) {
  return sizeof(__nv_bfloat16) * (kRcTokens * (4 * static_cast<size_t>(d + 8) + (e + 8)) + kRcEarly * 32 * static_cast<size_t>(e + 8));
}

template <int NT>
static int launch_retention_output(const RetentionChunkParams& p, int chunks, cudaStream_t s) {
  const size_t smem = rc_output_smem(p.d, p.e);
  auto kern = p.e == 16 * NT ? retention_chunk_output_kernel<NT, true> : retention_chunk_output_kernel<NT, false>;
  LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared));
  kern<<<dim3(chunks, p.nh), 256, smem, s>>>(p);
  return 0;
}

}  // namespace llmctl

using namespace llmctl;

// q, k: [tokens, H d]; v: [tokens, H e]; freq: fp32 [rot / 2]; decay_m1: fp32 [H], decay minus one.
LLMCTL_API int llmctl_retention_prepare(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                                        const int* positions, const float* freq, int rot, const float* decay_m1, int tokens, float* work,
                                        int H, int d, int e, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && d > 0 && d <= 256 && e > 0 && rot >= 0 && rot <= d && rot % 2 == 0 && (rot == 0 || freq) && decay_m1 && work != nullptr);
  LLMCTL_REQUIRE((reinterpret_cast<uintptr_t>(work) & 15) == 0);
  if (tokens == 0) return 0;
  const RetentionPrepParams p{q, k, v, ldq, ldk, ldv, positions, freq, decay_m1, H, d, e, rot, ms_work(work, tokens, H, H, d, e, 3)};
  const int dp = ms_pad_rows(d);
  const dim3 grid(tokens, tokens < kNumSMs && H > 8 ? (H + 7) / 8 : 1);
  cudaStream_t s = (cudaStream_t)stream;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    if (dp == 32) retention_prepare_kernel<T, 1><<<grid, 256, 0, s>>>(p);
    else if (dp == 64) retention_prepare_kernel<T, 2><<<grid, 256, 0, s>>>(p);
    else if (dp == 128) retention_prepare_kernel<T, 4><<<grid, 256, 0, s>>>(p);
    else retention_prepare_kernel<T, 8><<<grid, 256, 0, s>>>(p);
  });
  LLMCTL_RETURN_LAST();
}

// work: filled by llmctl_retention_prepare with the same sizes; out: fp32 [tokens, H e].
LLMCTL_API int llmctl_retention_scan(float* work, const int* portions, int nportions, int tokens, float* state, float* out, int H, int d, int e,
                                     void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && d > 0 && d <= 256 && e > 0 && work != nullptr && (reinterpret_cast<uintptr_t>(work) & 15) == 0);
  if (nportions == 0 || tokens == 0) return 0;
  MatrixScanParams p{ms_work(work, tokens, H, H, d, e, 3), portions, state, out, H, H, d, e, ScanTail{nullptr, 0, 0, 0, 1, nullptr}};
  const int rc = dispatch_matrix_scan<3>(p, nportions, (cudaStream_t)stream);
  if (rc) return rc;
  LLMCTL_RETURN_LAST();
}

// Retention (kind 3) for portions of one token each: rotation, state update, read-out, the head's RMS norm (no weight) and gate.
LLMCTL_API int llmctl_retention_step(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                                     const int* positions, const float* freq, int rot, const float* decay_m1, const int* portions,
                                     int nportions, float* state, const void* gate, long long ldg, int gate_kind, float eps, void* out, int H,
                                     int d, int e, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && d > 0 && d <= 256 && e > 0 && q && k && v && decay_m1 && gate && rot >= 0 && rot <= d && rot % 2 == 0 && (rot == 0 || freq));
  if (nportions == 0) return 0;
  MatrixStepParams p{nullptr, q, k, v, 0, ldq, ldk, ldv, nullptr, nullptr, 1, nullptr, 0, nullptr, decay_m1, nullptr, nullptr, 0, portions, state,
                     nullptr, 0, gate, ldg, gate_kind, eps, out, H, H, d, e, positions, freq, rot};
  int rc = 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (rc = dispatch_matrix_step<T, 3>(p, nportions, (cudaStream_t)stream)));
  if (rc) return rc;
  LLMCTL_RETURN_LAST();
}

// 1 when bf16 prompts of these sizes run in chunks: d and e multiples of 16 up to 256, pairs in groups of four.
LLMCTL_API int llmctl_retention_chunked_ok(int d, int e, int rot) {
  return (d > 0 && e > 0 && d % 16 == 0 && e % 16 == 0 && d <= 256 && e <= 256 && rot % 8 == 0 && rot <= d && rc_output_smem(d, e) <= 220 * 1024) ? 1 : 0;
}

// bf16 only; rows of q, k, v and gate start at 16-byte boundaries.  tiles: the 64-token tiles of all portions, in order; cs: fp32
// scratch [tokens, rot]; scratch: fp32 [chunks, heads_per_pass, d, e].  out: [tokens, H e], normed and gated.
LLMCTL_API int llmctl_retention_chunked(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                                        const int* positions, const float* freq, int rot, const float* decay_m1, const int* portions,
                                        int nportions, const int* tiles, int chunks, int tokens, float* state, const void* gate, long long ldg,
                                        int gate_kind, float eps, float* cs, float* scratch, int heads_per_pass, void* out, int H, int d, int e,
                                        void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(llmctl_retention_chunked_ok(d, e, rot) && H > 0 && heads_per_pass > 0 && decay_m1 && scratch && (rot == 0 || (freq && cs)));
  LLMCTL_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(gate) |
                   reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(scratch) | reinterpret_cast<uintptr_t>(cs) | reinterpret_cast<uintptr_t>(out)) & 15) == 0 &&
                 ldq % 8 == 0 && ldk % 8 == 0 && ldv % 8 == 0 && ldg % 8 == 0);
  if (chunks == 0 || tokens == 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  RetentionChunkParams p{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, (const __nv_bfloat16*)gate, ldq, ldk, ldv, ldg,
                         (const float2*)cs, rot / 2, decay_m1, portions, nportions, tiles, state, scratch, (__nv_bfloat16*)out, H, d, e, 0, 0,
                         gate_kind, eps};
  if (rot > 0) retention_angles_kernel<<<(tokens * (rot / 2) + 255) / 256, 256, 0, s>>>(positions, freq, rot / 2, (float2*)cs, tokens);
  const size_t smem = rc_sum_smem(d, e);
  LLMCTL_CHECK(cudaFuncSetAttribute(retention_chunk_sum_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  LLMCTL_CHECK(cudaFuncSetAttribute(retention_chunk_sum_kernel, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared));
  for (int h0 = 0; h0 < H; h0 += heads_per_pass) {
    p.h0 = h0;
    p.nh = H - h0 < heads_per_pass ? H - h0 : heads_per_pass;
    retention_chunk_sum_kernel<<<dim3(chunks, p.nh), 256, smem, s>>>(p);
    retention_chunk_chain_kernel<<<dim3(nportions, p.nh, (d * e / 8 + 255) / 256), 256, 0, s>>>(p);
    const int nt = (e / 8 + 1) / 2;
    const int rc = nt <= 2 ? launch_retention_output<2>(p, chunks, s) : nt <= 4 ? launch_retention_output<4>(p, chunks, s)
                 : nt <= 8 ? launch_retention_output<8>(p, chunks, s) : launch_retention_output<16>(p, chunks, s);
    if (rc) return rc;
  }
  LLMCTL_RETURN_LAST();
}
