// Recurrences with a matrix state per head, for ragged batches (portions of prompts next to single decoded tokens), bf16 or
// fp32 projections.  S: [d, e] fp32 per head, zero before a sequence's first token, kept in the sequence's state slot.
//
//   Gated delta rule (kinds 0 and 1), q and k unit vectors per key/value head (G of them; head h reads h / (H / G)):
//
//       q, k, v   = silu(causal convolution over time of the projections);   q <- q / |q| / sqrt(d), k <- k / |k|
//       g         = exp(-exp(A_h) softplus(z + dt_bias))       kind 0: one z per head; kind 1: one per head and key row
//       S <- g S;   u = beta (v - S^T k), beta = sigmoid(b);   S <- S + k u^T;   o = S^T q
//
//   Decayed outer products with a bonus for the current token (kind 2, d == e, G == H):
//
//       o = S^T r + (sum_i r_i u_i k_i) v;   S <- diag(w) S + k v^T,   w = exp(-exp(z + w0)) per head and key row
//
//   llmctl_delta_prepare / llmctl_bonus_prepare : fully parallel over tokens: convolutions, unit norms, step sizes, decays
//       (minus one) and the per-token scalars, in fp32 and padded so that the scan copies whole 16-byte rows.
//   llmctl_matrix_scan : the serial part.  A CTA owns (portion, head, 32 value columns).  LPC lanes share two columns, each
//       with d / LPC rows of both in registers; a token costs one pass over them (decay, S^T k and S^T q together: the
//       read-out after the write is S_before^T q + (q . k) u), log2(LPC) shuffles and one update.  Products run as packed
//       pairs (fma.rn.f32x2).  Chunks of 16 tokens are double-buffered in shared memory by cp.async.  At the end the CTAs of a
//       portion also store its last raw inputs (the convolution's, or the previous token's row for kind 2's token shift).
//   llmctl_matrix_step : one decoded token per sequence in ONE launch: convolution, norms, decays, state update, read-out,
//       the head's RMS norm and output gate.  A CTA owns (sequence, key/value head) and streams the states of its heads
//       through registers once.
// The decay is applied as S + (g - 1) S with g - 1 from expm1: slow decays keep their precision.
// Everything here is fp32; only the projections and the gated output have the activation type.
// Reference: none (the reference has no model code).
#include "../common/dtype.cuh"
#include "../common/mma_sync.cuh"

namespace llmctl {

__device__ __forceinline__ float ms_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float ms_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float ms_silu(float x) { return x / (1.f + expf(-x)); }

constexpr int kMsTC = 16;           // tokens per staged chunk of the scan
constexpr int kMsCols = 32;         // value columns per CTA of the scan
constexpr int kMsWalk = 16;         // consecutive tokens a warp of the prepare kernels walks

static inline __host__ __device__ int ms_pad_rows(int d) { return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256; }
static inline __host__ __device__ int ms_pad_cols(int e) { return (e + kMsCols - 1) / kMsCols * kMsCols; }

// ---------------------------------------------------------------------------------------------------------------
// prepare
// ---------------------------------------------------------------------------------------------------------------
struct MsWork {         // fp32 scratch of a step's tokens
  float* q;             // [T, G, dp]
  float* k;             // [T, G, dp]
  float* v;             // [T, H, ep]
  float* dm;            // [T, H, dp] decays minus one (kinds 1 and 2)
  float* sc;            // [T, H, 4] = (beta, q . k or the bonus, decay minus one of kind 0, 0)
};

struct DeltaPrepParams {
  const void* x;              // [T, ldx] raw [q | k | v]: C = 2 G d + H e columns
  long long ldx;
  const float* conv_w;        // [C, taps], last column = the current token's
  const float* conv_state;    // [slots, taps - 1, C]
  const void* z;              // decay projection: [T, H] (kind 0) or [T, H d] (kind 1)
  long long ldz;
  const float* dt_bias;       // like z
  const float* speed;         // [H] exp(A)
  const void* b;              // [T, H] write-strength logits
  long long ldb;
  const int* portions;
  const int* seq_rows;
  int T, H, G, d, e, taps, kind;
  MsWork w;
};

// raw input of channel c at token row src (< t0: from the state slot's rows, zeros before the sequence)
template <typename T>
__device__ __forceinline__ float ms_raw(const T* x, long long ldx, long long src, int t0, const float* st, int keep, int C, int c) {
  if (src >= t0) return to_f32(x[src * ldx + c]);
  return st ? st[static_cast<long long>(keep - (t0 - src)) * C + c] : 0.f;
}

// Short convolution of one channel along consecutive tokens: up to four taps keep weights and history in registers,
// longer ones read every tap again.
template <typename T>
struct ConvWalk {
  float w[4], h[3];
  __device__ __forceinline__ void weights(const float* conv_w, int taps, int c) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int src = taps - 4 + j;                   // w[3] is the current token's weight
      w[j] = (taps <= 4 && src >= 0) ? conv_w[static_cast<long long>(c) * taps + src] : 0.f;
    }
  }
  __device__ __forceinline__ void history(const T* x, long long ldx, long long t, int t0, const float* st, int taps, int C, int c) {
#pragma unroll
    for (int j = 0; j < 3; ++j) {
      const int back = 3 - j;
      h[j] = back <= taps - 1 ? ms_raw(x, ldx, t - back, t0, st, taps - 1, C, c) : 0.f;
    }
  }
  __device__ __forceinline__ float step(const T* x, long long ldx, long long t, int t0, const float* st, const float* conv_w, int taps,
                                        int C, int c) {
    const float cur = to_f32(x[t * ldx + c]);
    float a;
    if (taps <= 4) {
      a = w[0] * h[0] + w[1] * h[1] + w[2] * h[2] + w[3] * cur;
      h[0] = h[1];
      h[1] = h[2];
      h[2] = cur;
    } else {
      a = conv_w[static_cast<long long>(c) * taps + taps - 1] * cur;
      for (int j = 0; j < taps - 1; ++j)
        a += conv_w[static_cast<long long>(c) * taps + j] * ms_raw(x, ldx, t - (taps - 1 - j), t0, st, taps - 1, C, c);
    }
    return ms_silu(a);
  }
};

// A warp is one unit: units 0 .. G-1 are the query and key of a key/value head, then blocks of 128 padded value columns,
// then (kind 1) blocks of 128 padded decay columns.  blockIdx.x: a walk of kMsWalk tokens.
template <typename T, int NI>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaPrepParams p) {
  const int lane = threadIdx.x & 31;
  const int H = p.H, G = p.G, d = p.d, e = p.e, taps = p.taps, keep = taps - 1;
  const int dp = ms_pad_rows(d), ep = ms_pad_cols(e), rep = H / G, C = 2 * G * d + H * e;
  const int nv = (H * ep + 127) / 128, nd = p.kind == 1 ? (H * dp + 127) / 128 : 0;
  int unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (unit >= G + nv + nd) return;
  const int tb = blockIdx.x * kMsWalk, te = min(tb + kMsWalk, p.T);
  const T* x = static_cast<const T*>(p.x);
  int prow = -1, t0 = 0;
  const float* st = nullptr;
  auto enter = [&](int t) {               // true when token t opens a portion (or the walk): histories are stale
    const int r = p.seq_rows[t];
    if (r == prow) return false;
    prow = r;
    const int* pt = p.portions + 4 * r;
    t0 = pt[0];
    st = (pt[2] > 0 && pt[3] >= 0) ? p.conv_state + static_cast<long long>(pt[3]) * keep * C : nullptr;
    return true;
  };
  if (unit < G) {
    const int g = unit;
    ConvWalk<T> cq[NI], ck[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = lane + 32 * i;
      if (c < d) {
        cq[i].weights(p.conv_w, taps, g * d + c);
        ck[i].weights(p.conv_w, taps, (G + g) * d + c);
      }
    }
    const float qs = rsqrtf(static_cast<float>(d));
    for (int t = tb; t < te; ++t) {
      const bool fresh = enter(t);
      float q[NI], k[NI], sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int c = lane + 32 * i;
        q[i] = k[i] = 0.f;
        if (c < d) {
          if (fresh && taps <= 4) {
            cq[i].history(x, p.ldx, t, t0, st, taps, C, g * d + c);
            ck[i].history(x, p.ldx, t, t0, st, taps, C, (G + g) * d + c);
          }
          q[i] = cq[i].step(x, p.ldx, t, t0, st, p.conv_w, taps, C, g * d + c);
          k[i] = ck[i].step(x, p.ldx, t, t0, st, p.conv_w, taps, C, (G + g) * d + c);
        }
        sq += q[i] * q[i];
        sk += k[i] * k[i];
        qk += q[i] * k[i];
      }
      const float fq = qs / sqrtf(warp_sum(sq) + 1e-6f), fk = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
      qk = warp_sum(qk) * fq * fk;
      float* wq = p.w.q + (static_cast<long long>(t) * G + g) * dp;
      float* wk = p.w.k + (static_cast<long long>(t) * G + g) * dp;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        wq[lane + 32 * i] = q[i] * fq;
        wk[lane + 32 * i] = k[i] * fk;
      }
      for (int r = lane; r < rep; r += 32) {
        const int h = g * rep + r;
        const float beta = ms_sigmoid(to_f32(static_cast<const T*>(p.b)[static_cast<long long>(t) * p.ldb + h]));
        float dm = 0.f;
        if (p.kind == 0) dm = expm1f(-p.speed[h] * ms_softplus(to_f32(static_cast<const T*>(p.z)[static_cast<long long>(t) * p.ldz + h]) + p.dt_bias[h]));
        *reinterpret_cast<float4*>(p.w.sc + (static_cast<long long>(t) * H + h) * 4) = make_float4(beta, qk, dm, 0.f);
      }
    }
    return;
  }
  unit -= G;
  if (unit < nv) {
    ConvWalk<T> cv[4];
    int ch[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int col = unit * 128 + lane + 32 * i, h = col / ep, c = col % ep;
      ch[i] = (h < H && c < e) ? 2 * G * d + h * e + c : -1;
      if (ch[i] >= 0) cv[i].weights(p.conv_w, taps, ch[i]);
    }
    for (int t = tb; t < te; ++t) {
      const bool fresh = enter(t);
      float* wv = p.w.v + static_cast<long long>(t) * H * ep + unit * 128 + lane;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float v = 0.f;
        if (ch[i] >= 0) {
          if (fresh && taps <= 4) cv[i].history(x, p.ldx, t, t0, st, taps, C, ch[i]);
          v = cv[i].step(x, p.ldx, t, t0, st, p.conv_w, taps, C, ch[i]);
        }
        if (unit * 128 + lane + 32 * i < H * ep) wv[32 * i] = v;
      }
    }
    return;
  }
  unit -= nv;
  int zc[4];
  float sp[4], bias[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int col = unit * 128 + lane + 32 * i, h = col / dp, c = col % dp;
    const bool ok = h < H && c < d;
    zc[i] = ok ? h * d + c : -1;
    sp[i] = ok ? p.speed[h] : 0.f;
    bias[i] = ok ? p.dt_bias[zc[i]] : 0.f;
  }
  for (int t = tb; t < te; ++t) {
    float* wd = p.w.dm + static_cast<long long>(t) * H * dp + unit * 128 + lane;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float v = 0.f;
      if (zc[i] >= 0) v = expm1f(-sp[i] * ms_softplus(to_f32(static_cast<const T*>(p.z)[static_cast<long long>(t) * p.ldz + zc[i]]) + bias[i]));
      if (unit * 128 + lane + 32 * i < H * dp) wd[32 * i] = v;
    }
  }
}

struct BonusPrepParams {
  const void* r;              // [T, H d] each (row strides below)
  const void* k;
  const void* v;
  const void* z;              // decay projection
  long long ldr, ldk, ldv, ldz;
  const float* w0;            // [H d] decay offset
  const float* u;             // [H d] bonus
  int T, H, d;
  MsWork w;
};

// one warp per (token, head)
template <typename T, int NI>
__global__ void __launch_bounds__(256)
bonus_prepare_kernel(const BonusPrepParams p) {
  const int lane = threadIdx.x & 31, H = p.H, d = p.d;
  const int dp = ms_pad_rows(d), ep = ms_pad_cols(d);
  const long long rows = static_cast<long long>(p.T) * H;
  for (long long row = blockIdx.x * 8LL + (threadIdx.x >> 5); row < rows; row += gridDim.x * 8LL) {
    const long long t = row / H;
    const int h = static_cast<int>(row % H);
    float bonus = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = lane + 32 * i, col = h * d + c;
      float r = 0.f, k = 0.f, v = 0.f, dm = 0.f;
      if (c < d) {
        r = to_f32(static_cast<const T*>(p.r)[t * p.ldr + col]);
        k = to_f32(static_cast<const T*>(p.k)[t * p.ldk + col]);
        v = to_f32(static_cast<const T*>(p.v)[t * p.ldv + col]);
        dm = expm1f(-expf(to_f32(static_cast<const T*>(p.z)[t * p.ldz + col]) + p.w0[col]));
        bonus += r * p.u[col] * k;
      }
      p.w.q[row * dp + c] = r;
      p.w.k[row * dp + c] = k;
      p.w.dm[row * dp + c] = dm;
      if (c < ep) p.w.v[row * ep + c] = v;
    }
    bonus = warp_sum(bonus);
    if (lane == 0) *reinterpret_cast<float4*>(p.w.sc + row * 4) = make_float4(1.f, bonus, 0.f, 0.f);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// scan
// ---------------------------------------------------------------------------------------------------------------
typedef unsigned long long f32x2;

__device__ __forceinline__ f32x2 pk(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 upk(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
// two neighbouring pairs from 16 aligned bytes of shared memory
__device__ __forceinline__ void ld_pairs(const float* s, f32x2& a, f32x2& b) {
  const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(s);
  a = v.x;
  b = v.y;
}

struct ScanTail {             // rows stored for the next portion: the last `keep` rows of x (older ones shift in)
  const void* x;              // [T, ldx], C columns used
  long long ldx;
  int C, keep, is32;
  float* state;               // [slots, keep, C]
};

struct MatrixScanParams {
  MsWork w;
  const int* portions;
  float* state;               // [slots, H, d, e]
  float* out;                 // [T, H, e]
  int H, G, d, e;
  ScanTail tail;
};

// KIND 0: delta rule, decay per head; 1: delta rule, decay per key row; 2: outer products with a bonus.
// A lane owns columns c0 and c0 + 1 and the rows (i LPC + sub) 4 .. + 3, i < RPT / 4.
template <int RPT, int LPC, int KIND>
__global__ void __launch_bounds__(LPC * 16)
matrix_scan_kernel(const MatrixScanParams p) {
  constexpr int TC = kMsTC, DP = RPT * LPC, NG = 32 / LPC, NT = LPC * 16, NP = RPT / 2;
  constexpr int STAGE = TC * (DP * (KIND == 0 ? 2 : 3) + kMsCols + 4);
  extern __shared__ __align__(16) float ms_smem[];
  const int H = p.H, d = p.d, e = p.e;
  const int* pt = p.portions + blockIdx.x * 4;
  const int t0 = pt[0], n = pt[1], pos0 = pt[2], slot = pt[3];
  if (n <= 0) return;
  const int h = blockIdx.y, kvh = h / (H / p.G), ep = ms_pad_cols(e), cb = blockIdx.z * kMsCols;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = lane % LPC;
  const int cl = (warp * NG + lane / LPC) * 2;               // first of this lane's columns within the CTA's
  float* so = ms_smem + 2 * STAGE;                           // [2][TC][32] outputs of the chunk

  f32x2 S[2][NP];
  float* st = slot >= 0 ? p.state + ((static_cast<long long>(slot) * H + h) * d) * e : nullptr;
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int row = ((j >> 1) * LPC + sub) * 4 + (j & 1) * 2, col = cb + cl + c;
      float a = 0.f, b = 0.f;
      if (st && pos0 > 0 && col < e) {
        if (row < d) a = st[static_cast<long long>(row) * e + col];
        if (row + 1 < d) b = st[static_cast<long long>(row + 1) * e + col];
      }
      S[c][j] = pk(a, b);
    }

  auto stage = [&](int c0, int buf) {                        // copies of tokens c0 .. c0 + TC - 1 into buffer buf
    float* sk = ms_smem + buf * STAGE;
    float* sq = sk + TC * DP;
    float* sd = sq + TC * DP;
    float* sv = sk + TC * DP * (KIND == 0 ? 2 : 3);
    float* ss = sv + TC * kMsCols;
    const int cnt = min(TC, n - c0);
    const long long tb = t0 + c0;
    for (int i = tid; i < cnt * (DP / 4); i += NT) {
      const int tok = i / (DP / 4), c = i % (DP / 4) * 4;
      const long long src = ((tb + tok) * p.G + kvh) * DP + c;
      cp_async_16(sk + tok * DP + c, p.w.k + src);
      cp_async_16(sq + tok * DP + c, p.w.q + src);
      if (KIND != 0) cp_async_16(sd + tok * DP + c, p.w.dm + ((tb + tok) * H + h) * DP + c);
    }
    for (int i = tid; i < cnt * 9; i += NT) {
      const int tok = i / 9, c = i % 9;
      if (c < 8) cp_async_16(sv + tok * kMsCols + c * 4, p.w.v + ((tb + tok) * H + h) * ep + cb + c * 4);
      else cp_async_16(ss + tok * 4, p.w.sc + ((tb + tok) * H + h) * 4);
    }
  };
  auto flush = [&](int c0, int buf) {                        // the chunk's outputs, 32 neighbouring columns per token
    const int cnt = min(TC, n - c0);
    for (int i = tid; i < cnt * kMsCols; i += NT) {
      const int tok = i / kMsCols, c = i % kMsCols;
      if (cb + c < e) p.out[(static_cast<long long>(t0 + c0 + tok) * H + h) * e + cb + c] = so[(buf * TC + tok) * kMsCols + c];
    }
  };

  stage(0, 0);
  cp_async_commit();
  int buf = 0;
  for (int c0 = 0; c0 < n; c0 += TC, buf ^= 1) {
    cp_async_wait_all();
    __syncthreads();                                         // the chunk has landed; everyone is done with the other buffers
    if (c0 + TC < n) stage(c0 + TC, buf ^ 1);
    cp_async_commit();
    if (c0 > 0) flush(c0 - TC, buf ^ 1);
    const float* sk = ms_smem + buf * STAGE + sub * 4;
    const float* sq = sk + TC * DP;
    const float* sd = sq + TC * DP;
    const float* sv = ms_smem + buf * STAGE + TC * DP * (KIND == 0 ? 2 : 3) + cl;
    const float* ss = ms_smem + buf * STAGE + TC * DP * (KIND == 0 ? 2 : 3) + TC * kMsCols;
    float* od = so + buf * TC * kMsCols + cl;
    const int cnt = min(TC, n - c0);
#pragma unroll 1
    for (int tok = 0; tok < cnt; ++tok) {
      f32x2 k[NP], ka0 = 0ull, ka1 = 0ull, kb0 = 0ull, kb1 = 0ull, qa0 = 0ull, qa1 = 0ull, qb0 = 0ull, qb1 = 0ull;
      const float4 sc = *reinterpret_cast<const float4*>(ss + tok * 4);
      const float2 v = *reinterpret_cast<const float2*>(sv + tok * kMsCols);
      const f32x2 dh = pk(sc.z, sc.z);
#pragma unroll
      for (int i = 0; i < NP; i += 2) {
        f32x2 q0, q1, d0 = dh, d1 = dh;
        ld_pairs(sk + tok * DP + i * 2 * LPC, k[i], k[i + 1]);
        ld_pairs(sq + tok * DP + i * 2 * LPC, q0, q1);
        if (KIND != 0) ld_pairs(sd + tok * DP + i * 2 * LPC, d0, d1);
        if (KIND == 2) {                                     // the read-out sees the state before this token
          qa0 = fma2(q0, S[0][i], qa0);
          qa1 = fma2(q1, S[0][i + 1], qa1);
          qb0 = fma2(q0, S[1][i], qb0);
          qb1 = fma2(q1, S[1][i + 1], qb1);
        }
        S[0][i] = fma2(d0, S[0][i], S[0][i]);
        S[0][i + 1] = fma2(d1, S[0][i + 1], S[0][i + 1]);
        S[1][i] = fma2(d0, S[1][i], S[1][i]);
        S[1][i + 1] = fma2(d1, S[1][i + 1], S[1][i + 1]);
        if (KIND != 2) {
          ka0 = fma2(k[i], S[0][i], ka0);
          ka1 = fma2(k[i + 1], S[0][i + 1], ka1);
          kb0 = fma2(k[i], S[1][i], kb0);
          kb1 = fma2(k[i + 1], S[1][i + 1], kb1);
          qa0 = fma2(q0, S[0][i], qa0);
          qa1 = fma2(q1, S[0][i + 1], qa1);
          qb0 = fma2(q0, S[1][i], qb0);
          qb1 = fma2(q1, S[1][i + 1], qb1);
        }
      }
      float ua = v.x, ub = v.y;
      if (KIND != 2) {
        const float2 a0 = upk(ka0), a1 = upk(ka1), b0 = upk(kb0), b1 = upk(kb1);
        float ka = (a0.x + a1.x) + (a0.y + a1.y), kb = (b0.x + b1.x) + (b0.y + b1.y);
#pragma unroll
        for (int o = LPC / 2; o > 0; o >>= 1) {
          ka += __shfl_xor_sync(0xffffffffu, ka, o);
          kb += __shfl_xor_sync(0xffffffffu, kb, o);
        }
        ua = sc.x * (v.x - ka);
        ub = sc.x * (v.y - kb);
      }
      const f32x2 u0 = pk(ua, ua), u1 = pk(ub, ub);
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        S[0][i] = fma2(k[i], u0, S[0][i]);
        S[1][i] = fma2(k[i], u1, S[1][i]);
      }
      const float2 a0 = upk(qa0), a1 = upk(qa1), b0 = upk(qb0), b1 = upk(qb1);
      float qa = (a0.x + a1.x) + (a0.y + a1.y), qb = (b0.x + b1.x) + (b0.y + b1.y);
#pragma unroll
      for (int o = LPC / 2; o > 0; o >>= 1) {
        qa += __shfl_xor_sync(0xffffffffu, qa, o);
        qb += __shfl_xor_sync(0xffffffffu, qb, o);
      }
      if (sub == 0) *reinterpret_cast<float2*>(od + tok * kMsCols) = make_float2(qa + sc.y * ua, qb + sc.y * ub);
    }
  }
  __syncthreads();
  flush((n - 1) / TC * TC, buf ^ 1);
  if (!st) return;
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int row = ((j >> 1) * LPC + sub) * 4 + (j & 1) * 2, col = cb + cl + c;
      const float2 s = upk(S[c][j]);
      if (col < e) {
        if (row < d) st[static_cast<long long>(row) * e + col] = s.x;
        if (row + 1 < d) st[static_cast<long long>(row + 1) * e + col] = s.y;
      }
    }
  // the CTAs of the portion share the columns of its last raw rows; a column belongs to one thread
  const ScanTail& tl = p.tail;
  if (tl.keep <= 0) return;
  float* ts = tl.state + static_cast<long long>(slot) * tl.keep * tl.C;
  for (int c = (h * gridDim.z + blockIdx.z) * NT + tid; c < tl.C; c += H * gridDim.z * NT)
    for (int j = 0; j < tl.keep; ++j) {                      // ascending: row j takes what row j + n held
      const int src = n - tl.keep + j;                       // token of the portion, negative: before it
      float v = 0.f;
      if (src >= 0) {
        const long long at = (t0 + src) * tl.ldx + c;
        v = tl.is32 ? static_cast<const float*>(tl.x)[at] : __bfloat162float(static_cast<const __nv_bfloat16*>(tl.x)[at]);
      } else if (pos0 > 0) {
        v = ts[static_cast<long long>(j + n) * tl.C + c];
      }
      ts[static_cast<long long>(j) * tl.C + c] = v;
    }
}

// ---------------------------------------------------------------------------------------------------------------
// one decoded token per sequence
// ---------------------------------------------------------------------------------------------------------------
struct MatrixStepParams {
  const void* x;              // kinds 0, 1: raw [q | k | v] (row stride ldx)
  const void* r;              // kind 2: r, k, v (row strides ldr, ldk, ldv)
  const void* k;
  const void* v;
  long long ldx, ldr, ldk, ldv;
  const float* conv_w;        // kinds 0, 1
  float* conv_state;
  int taps;
  const void* z;
  long long ldz;
  const float* z_bias;        // dt_bias, or w0 of kind 2
  const float* speed;         // [H], kinds 0, 1
  const float* bonus;         // [H d], kind 2
  const void* b;              // [T, H], kinds 0, 1
  long long ldb;
  const int* portions;
  float* state;               // [slots, H, d, e]
  const float* norm_w;        // [e] (norm_stride 0) or [H, e] (norm_stride e)
  int norm_stride;
  const void* gate;           // [T, H e] pre-activation
  long long ldg;
  int gate_kind;              // 0: silu, 1: sigmoid
  float eps;
  void* out;                  // [T, H e]
  int H, G, d, e;
};

template <typename T>
__device__ __forceinline__ float ms_conv_step(const T* x, const float* w, float* st, bool has, int taps, int C, int c) {
  // one token: history from the state rows, which then move on by one
  const float cur = to_f32(x[c]);
  float a = w[static_cast<long long>(c) * taps + taps - 1] * cur;
  for (int j = 0; j < taps - 1; ++j) {
    const float v = has ? st[static_cast<long long>(j) * C + c] : 0.f;
    a += w[static_cast<long long>(c) * taps + j] * v;
    if (st && j > 0) st[static_cast<long long>(j - 1) * C + c] = v;
  }
  if (st && taps > 1) st[static_cast<long long>(taps - 2) * C + c] = cur;
  return ms_silu(a);
}

template <int VEC>
__device__ __forceinline__ void ms_ldv(const float* p, float (&v)[VEC]) {
  if (VEC == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
  else v[0] = p[0];
}
template <int VEC>
__device__ __forceinline__ void ms_stv(float* p, const float (&v)[VEC]) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(v);
  else p[0] = v[0];
}

// 8 warps share the rows of S (RPW each), a lane VEC neighbouring columns of a tile of 32 VEC.
template <typename T, int RPW, int VEC, int KIND>
__global__ void __launch_bounds__(256, RPW * VEC <= 64 ? 2 : 1)
matrix_step_kernel(const MatrixStepParams p) {
  constexpr int DP = RPW * 8, TILE = 32 * VEC;
  extern __shared__ __align__(16) float ms_smem[];
  __shared__ float red[64];
  const int H = p.H, G = p.G, d = p.d, e = p.e, rep = H / G, g = blockIdx.y;
  const int* pt = p.portions + blockIdx.x * 4;
  const long long t = pt[0];
  const int slot = pt[3];
  if (pt[1] <= 0) return;
  const bool has = slot >= 0 && pt[2] > 0;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* sq = ms_smem;                 // [DP]
  float* sk = sq + DP;                 // [DP]
  float* sd = sk + DP;                 // [DP]
  float* part = sd + DP;               // [8][2][TILE] partial S^T k and S^T q of the warps
  float* sv = part + 16 * TILE;        // [e]
  float* so = sv + e;                  // [e]
  const int C = 2 * G * d + H * e;
  float* cst = (KIND != 2 && slot >= 0) ? p.conv_state + static_cast<long long>(slot) * (p.taps - 1) * C : nullptr;

  __align__(16) float S[RPW][VEC];
  auto load_state = [&](int h, int c0) {
    const float* st = p.state + (static_cast<long long>(slot) * H + h) * d * e;
    const int col = c0 + lane * VEC;
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int row = warp * RPW + i;
#pragma unroll
      for (int j = 0; j < VEC; ++j) S[i][j] = 0.f;
      if (has && row < d && col < e) ms_ldv<VEC>(st + static_cast<long long>(row) * e + col, S[i]);
    }
  };
  load_state(g * rep, 0);              // in flight while the token's vectors are formed

  float qk = 0.f;
  {
    float q = 0.f, k = 0.f;
    if (tid < d) {
      if (KIND == 2) {
        q = to_f32(static_cast<const T*>(p.r)[t * p.ldr + g * d + tid]);
        k = to_f32(static_cast<const T*>(p.k)[t * p.ldk + g * d + tid]);
      } else {
        const T* x = static_cast<const T*>(p.x) + t * p.ldx;
        q = ms_conv_step(x, p.conv_w, cst, has, p.taps, C, g * d + tid);
        k = ms_conv_step(x, p.conv_w, cst, has, p.taps, C, (G + g) * d + tid);
      }
    }
    if (KIND == 2) {
      qk = block_sum(tid < d ? q * k * p.bonus[g * d + tid] : 0.f, red);
    } else {
      const float fq = rsqrtf(static_cast<float>(d)) / sqrtf(block_sum(q * q, red) + 1e-6f);
      const float fk = 1.f / sqrtf(block_sum(k * k, red) + 1e-6f);
      q *= fq;
      k *= fk;
      qk = block_sum(q * k, red);
    }
    if (tid < DP) sq[tid] = q, sk[tid] = k;
  }
  for (int r = 0; r < rep; ++r) {
    const int h = g * rep + r;
    if (r > 0) {
      __syncthreads();                 // the previous head's readers of sv, so, sd are done
      load_state(h, 0);
    }
    float beta = 1.f, dm = 0.f;
    if (KIND != 2) {
      beta = ms_sigmoid(to_f32(static_cast<const T*>(p.b)[t * p.ldb + h]));
      if (KIND == 0) dm = expm1f(-p.speed[h] * ms_softplus(to_f32(static_cast<const T*>(p.z)[t * p.ldz + h]) + p.z_bias[h]));
    }
    if (KIND != 0 && tid < DP) {
      float v = 0.f;
      if (tid < d) {
        const float z = to_f32(static_cast<const T*>(p.z)[t * p.ldz + h * d + tid]) + p.z_bias[h * d + tid];
        v = KIND == 2 ? expm1f(-expf(z)) : expm1f(-p.speed[h] * ms_softplus(z));
      }
      sd[tid] = v;
    }
    for (int c = tid; c < e; c += 256) {
      if (KIND == 2) sv[c] = to_f32(static_cast<const T*>(p.v)[t * p.ldv + h * e + c]);
      else sv[c] = ms_conv_step(static_cast<const T*>(p.x) + t * p.ldx, p.conv_w, cst, has, p.taps, C, 2 * G * d + h * e + c);
    }
    __syncthreads();
    float* st = slot >= 0 ? p.state + (static_cast<long long>(slot) * H + h) * d * e : nullptr;
    for (int c0 = 0; c0 < e; c0 += TILE) {
      if (c0 > 0) load_state(h, c0);
      const int col = c0 + lane * VEC;
      __align__(16) float ka[VEC], qa[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) ka[j] = qa[j] = 0.f;
#pragma unroll
      for (int i = 0; i < RPW; ++i) {
        const int row = warp * RPW + i;
        const float kk = sk[row], qq = sq[row], dd = KIND == 0 ? dm : sd[row];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          if (KIND == 2) qa[j] += qq * S[i][j];
          S[i][j] = fmaf(dd, S[i][j], S[i][j]);
          if (KIND != 2) {
            ka[j] += kk * S[i][j];
            qa[j] += qq * S[i][j];
          }
        }
      }
      if (KIND != 2) ms_stv<VEC>(part + (warp * 2) * TILE + lane * VEC, ka);
      ms_stv<VEC>(part + (warp * 2 + 1) * TILE + lane * VEC, qa);
      __syncthreads();
      float u[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) u[j] = col + j < e ? sv[col + j] : 0.f;
      if (KIND != 2) {
        __align__(16) float s[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) s[j] = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
          __align__(16) float v[VEC];
          ms_ldv<VEC>(part + (w * 2) * TILE + lane * VEC, v);
#pragma unroll
          for (int j = 0; j < VEC; ++j) s[j] += v[j];
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) u[j] = beta * (u[j] - s[j]);
      }
#pragma unroll
      for (int i = 0; i < RPW; ++i) {
        const int row = warp * RPW + i;
        const float kk = sk[row];
#pragma unroll
        for (int j = 0; j < VEC; ++j) S[i][j] = fmaf(kk, u[j], S[i][j]);
        if (st && row < d && col < e) ms_stv<VEC>(st + static_cast<long long>(row) * e + col, S[i]);
      }
      if (warp == 0) {
#pragma unroll
        for (int w = 0; w < 8; ++w) {
          __align__(16) float v[VEC];
          ms_ldv<VEC>(part + (w * 2 + 1) * TILE + lane * VEC, v);
#pragma unroll
          for (int j = 0; j < VEC; ++j)
            if (w == 0) qa[j] = v[j];
            else qa[j] += v[j];
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j)
          if (col + j < e) so[col + j] = qa[j] + qk * u[j];
      }
      __syncthreads();                 // so is complete; the partials are free
    }
    float ss = 0.f;
    for (int c = tid; c < e; c += 256) ss += so[c] * so[c];
    const float f = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(e) + p.eps);
    for (int c = tid; c < e; c += 256) {
      const float gz = to_f32(static_cast<const T*>(p.gate)[t * p.ldg + h * e + c]);
      const float act = p.gate_kind == 1 ? ms_sigmoid(gz) : ms_silu(gz);
      static_cast<T*>(p.out)[(t * H + h) * e + c] = from_f32<T>(so[c] * f * p.norm_w[h * p.norm_stride + c] * act);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------
// token shift
// ---------------------------------------------------------------------------------------------------------------
// out[s, t] = h[t] + (h[t - 1] - h[t]) * mu[s] for n_mix mixes; row -1 of a portion is the slot's stored row (zeros at
// position 0).  A portion of one token also stores its row; longer portions leave that to the scan that follows (a block
// must not overwrite a row that another block of this launch still reads).
template <typename T>
__global__ void __launch_bounds__(256)
token_shift_kernel(const T* __restrict__ h, const float* __restrict__ mu, int n_mix, const int* __restrict__ portions,
                   const int* __restrict__ seq_rows, float* __restrict__ state, T* __restrict__ out, int tokens, int W) {
  const long long t = blockIdx.x;
  const int* pt = portions + 4 * seq_rows[t];
  const int slot = pt[3];
  float* st = slot >= 0 ? state + static_cast<long long>(slot) * W : nullptr;
  const bool first = t == pt[0], has = st != nullptr && pt[2] > 0, store = first && pt[1] == 1 && st != nullptr;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float cur = to_f32(h[t * W + c]);
    float prev = 0.f;
    if (!first) prev = to_f32(h[(t - 1) * W + c]);
    else if (has) prev = st[c];
    if (store) st[c] = cur;
    for (int s = 0; s < n_mix; ++s) out[(static_cast<long long>(s) * tokens + t) * W + c] = from_f32<T>(cur + (prev - cur) * mu[s * W + c]);
  }
}

// four neighbouring columns per thread (W a multiple of 4, aligned rows)
template <typename T>
__device__ __forceinline__ float4 ms_ld4(const T* p);
template <>
__device__ __forceinline__ float4 ms_ld4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <>
__device__ __forceinline__ float4 ms_ld4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void ms_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ms_st4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

template <typename T>
__global__ void __launch_bounds__(256)
token_shift_vec_kernel(const T* __restrict__ h, const float* __restrict__ mu, int n_mix, const int* __restrict__ portions,
                       const int* __restrict__ seq_rows, float* __restrict__ state, T* __restrict__ out, int tokens, int W) {
  const long long t = blockIdx.x;
  const int* pt = portions + 4 * seq_rows[t];
  const int slot = pt[3];
  float* st = slot >= 0 ? state + static_cast<long long>(slot) * W : nullptr;
  const bool first = t == pt[0], has = st != nullptr && pt[2] > 0, store = first && pt[1] == 1 && st != nullptr;
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) << 2; c < W; c += (gridDim.y * blockDim.x) << 2) {
    const float4 cur = ms_ld4(h + t * W + c);
    float4 prev = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!first) prev = ms_ld4(h + (t - 1) * W + c);
    else if (has) prev = ms_ld4(st + c);
    if (store) ms_st4(st + c, cur);
    const float4 df = make_float4(prev.x - cur.x, prev.y - cur.y, prev.z - cur.z, prev.w - cur.w);
    for (int s = 0; s < n_mix; ++s) {
      const float4 m = ms_ld4(mu + static_cast<long long>(s) * W + c);
      ms_st4(out + (static_cast<long long>(s) * tokens + t) * W + c,
             make_float4(cur.x + df.x * m.x, cur.y + df.y * m.y, cur.z + df.z * m.z, cur.w + df.w * m.w));
    }
  }
}

template <int RPT, int LPC, int KIND>
static int launch_matrix_scan(const MatrixScanParams& p, int nportions, cudaStream_t s) {
  constexpr int DP = RPT * LPC;
  const size_t smem = sizeof(float) * (2 * kMsTC * (static_cast<size_t>(DP) * (KIND == 0 ? 2 : 3) + kMsCols + 4) + 2 * kMsTC * kMsCols);
  auto kern = matrix_scan_kernel<RPT, LPC, KIND>;
  if (smem > 48 * 1024) LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kern<<<dim3(nportions, p.H, ms_pad_cols(p.e) / kMsCols), LPC * 16, smem, s>>>(p);
  return 0;
}

template <int KIND>
static int dispatch_matrix_scan(const MatrixScanParams& p, int nportions, cudaStream_t s) {
  switch (ms_pad_rows(p.d)) {
    case 32: return launch_matrix_scan<8, 4, KIND>(p, nportions, s);
    case 64: return launch_matrix_scan<8, 8, KIND>(p, nportions, s);
    case 128: return launch_matrix_scan<16, 8, KIND>(p, nportions, s);
    default: return launch_matrix_scan<32, 8, KIND>(p, nportions, s);
  }
}

template <typename T, int RPW, int KIND>
static int launch_matrix_step(const MatrixStepParams& p, int nportions, cudaStream_t s) {
  const int vec = p.e % 4 == 0 ? 4 : 1;
  const size_t smem = sizeof(float) * (3 * RPW * 8 + 16 * 32 * static_cast<size_t>(vec) + 2 * static_cast<size_t>(p.e));
  LLMCTL_REQUIRE(smem <= 48 * 1024);
  const dim3 grid(nportions, p.G);
  if (vec == 4) matrix_step_kernel<T, RPW, 4, KIND><<<grid, 256, smem, s>>>(p);
  else matrix_step_kernel<T, RPW, 1, KIND><<<grid, 256, smem, s>>>(p);
  return 0;
}

template <typename T, int KIND>
static int dispatch_matrix_step(const MatrixStepParams& p, int nportions, cudaStream_t s) {
  switch (ms_pad_rows(p.d)) {
    case 32: return launch_matrix_step<T, 4, KIND>(p, nportions, s);
    case 64: return launch_matrix_step<T, 8, KIND>(p, nportions, s);
    case 128: return launch_matrix_step<T, 16, KIND>(p, nportions, s);
    default: return launch_matrix_step<T, 32, KIND>(p, nportions, s);
  }
}

static MsWork ms_work(float* base, long long T, int H, int G, int d, int e, int kind) {
  const long long dp = ms_pad_rows(d), ep = ms_pad_cols(e);
  MsWork w;
  w.q = base;
  w.k = w.q + T * G * dp;
  w.v = w.k + T * G * dp;
  w.sc = w.v + T * H * ep;
  w.dm = w.sc + T * H * 4;
  return w;
}

}  // namespace llmctl

using namespace llmctl;

// fp32 numbers of scratch that the prepare and scan entry points need for `tokens` tokens
LLMCTL_API long long llmctl_matrix_scan_work(int tokens, int H, int G, int d, int e, int kind) {
  const long long dp = ms_pad_rows(d), ep = ms_pad_cols(e), T = tokens;
  return T * (2LL * G * dp + H * ep + 4LL * H + (kind == 0 ? 0 : H * dp));
}

// kind 0: z [tokens, H], dt_bias [H]; kind 1: z [tokens, H d], dt_bias [H d].  x: raw [q | k | v] columns.
LLMCTL_API int llmctl_delta_prepare(const void* x, long long ldx, const float* conv_w, const float* conv_state, int taps, const void* z,
                                    long long ldz, const float* dt_bias, const float* speed, const void* b, long long ldb,
                                    const int* portions, const int* seq_rows, int tokens, float* work, int H, int G, int d, int e,
                                    int kind, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && d <= 256 && e > 0 && taps >= 1 && (kind == 0 || kind == 1) && work != nullptr);
  LLMCTL_REQUIRE((reinterpret_cast<uintptr_t>(work) & 15) == 0 && (taps == 1 || conv_state != nullptr));
  if (tokens == 0) return 0;
  DeltaPrepParams p{x, ldx, conv_w, conv_state, z, ldz, dt_bias, speed, b, ldb, portions, seq_rows, tokens, H, G, d, e, taps, kind,
                    ms_work(work, tokens, H, G, d, e, kind)};
  const int dp = ms_pad_rows(d), ep = ms_pad_cols(e);
  const int units = G + (H * ep + 127) / 128 + (kind == 1 ? (H * dp + 127) / 128 : 0);
  const dim3 grid((tokens + kMsWalk - 1) / kMsWalk, (units + 7) / 8);
  cudaStream_t s = (cudaStream_t)stream;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    if (dp == 32) delta_prepare_kernel<T, 1><<<grid, 256, 0, s>>>(p);
    else if (dp == 64) delta_prepare_kernel<T, 2><<<grid, 256, 0, s>>>(p);
    else if (dp == 128) delta_prepare_kernel<T, 4><<<grid, 256, 0, s>>>(p);
    else delta_prepare_kernel<T, 8><<<grid, 256, 0, s>>>(p);
  });
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_bonus_prepare(const void* r, long long ldr, const void* k, long long ldk, const void* v, long long ldv, const void* z,
                                    long long ldz, const float* w0, const float* u, int tokens, float* work, int H, int d, int is_fp32,
                                    void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && d > 0 && d <= 256 && work != nullptr && (reinterpret_cast<uintptr_t>(work) & 15) == 0);
  if (tokens == 0) return 0;
  BonusPrepParams p{r, k, v, z, ldr, ldk, ldv, ldz, w0, u, tokens, H, d, ms_work(work, tokens, H, H, d, d, 2)};
  const long long rows = (static_cast<long long>(tokens) * H + 7) / 8;
  const int grid = static_cast<int>(rows < kNumSMs * 16LL ? rows : kNumSMs * 16LL);
  const int dp = ms_pad_rows(d);
  cudaStream_t s = (cudaStream_t)stream;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    if (dp == 32) bonus_prepare_kernel<T, 1><<<grid, 256, 0, s>>>(p);
    else if (dp == 64) bonus_prepare_kernel<T, 2><<<grid, 256, 0, s>>>(p);
    else if (dp == 128) bonus_prepare_kernel<T, 4><<<grid, 256, 0, s>>>(p);
    else bonus_prepare_kernel<T, 8><<<grid, 256, 0, s>>>(p);
  });
  LLMCTL_RETURN_LAST();
}

// work: filled by a prepare call with the same sizes; out: fp32 [tokens, H e]; the tail: last tail_keep rows of tail_x
// ([tokens, tail_ld], tail_C columns) into tail_state ([slots, tail_keep, tail_C] fp32).
LLMCTL_API int llmctl_matrix_scan(float* work, const int* portions, int nportions, int tokens, float* state, float* out, int H, int G, int d,
                                  int e, int kind, const void* tail_x, long long tail_ld, int tail_C, int tail_keep, float* tail_state,
                                  int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && d <= 256 && e > 0 && kind >= 0 && kind <= 2 && work != nullptr);
  LLMCTL_REQUIRE((reinterpret_cast<uintptr_t>(work) & 15) == 0 && (kind != 2 || (G == H && d == e)));
  LLMCTL_REQUIRE(tail_keep == 0 || (tail_x != nullptr && tail_state != nullptr && tail_ld >= tail_C));
  if (nportions == 0 || tokens == 0) return 0;
  MatrixScanParams p{ms_work(work, tokens, H, G, d, e, kind), portions, state, out, H, G, d, e,
                     ScanTail{tail_x, tail_ld, tail_C, tail_keep, is_fp32, tail_state}};
  cudaStream_t s = (cudaStream_t)stream;
  const int rc = kind == 0 ? dispatch_matrix_scan<0>(p, nportions, s) : kind == 1 ? dispatch_matrix_scan<1>(p, nportions, s)
                                                                                  : dispatch_matrix_scan<2>(p, nportions, s);
  if (rc) return rc;
  LLMCTL_RETURN_LAST();
}

// Every portion holds one token.  kinds 0, 1: x raw [q | k | v], conv_w, conv_state (updated), b, speed; kind 2: r, k, v, bonus.
// norm_stride: 0 (one weight vector of e numbers for all heads) or e.  gate_kind 0: silu, 1: sigmoid.
LLMCTL_API int llmctl_matrix_step(const void* x, long long ldx, const void* r, long long ldr, const void* k, long long ldk, const void* v,
                                  long long ldv, const float* conv_w, float* conv_state, int taps, const void* z, long long ldz,
                                  const float* z_bias, const float* speed, const float* bonus, const void* b, long long ldb,
                                  const int* portions, int nportions, float* state, const float* norm_w, int norm_stride,
                                  const void* gate, long long ldg, int gate_kind, float eps, void* out, int H, int G, int d, int e,
                                  int kind, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && d <= 256 && e > 0 && kind >= 0 && kind <= 2 && (kind != 2 || (G == H && d == e)));
  LLMCTL_REQUIRE(kind == 2 ? (r && k && v && bonus) : (x && conv_w && b && speed && taps >= 1 && (taps == 1 || conv_state)));
  if (nportions == 0) return 0;
  MatrixStepParams p{x, r, k, v, ldx, ldr, ldk, ldv, conv_w, conv_state, taps, z, ldz, z_bias, speed, bonus, b, ldb, portions, state,
                     norm_w, norm_stride, gate, ldg, gate_kind, eps, out, H, G, d, e};
  cudaStream_t s = (cudaStream_t)stream;
  int rc = 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    rc = kind == 0 ? dispatch_matrix_step<T, 0>(p, nportions, s) : kind == 1 ? dispatch_matrix_step<T, 1>(p, nportions, s)
                                                                             : dispatch_matrix_step<T, 2>(p, nportions, s);
  });
  if (rc) return rc;
  LLMCTL_RETURN_LAST();
}

// h: [tokens, W] contiguous; mu: fp32 [n_mix, W]; state: fp32 [slots, W]; out: [n_mix, tokens, W].
LLMCTL_API int llmctl_token_shift(const void* h, const float* mu, int n_mix, const int* portions, const int* seq_rows, float* state,
                                  void* out, int tokens, int W, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(W > 0 && n_mix > 0);
  if (tokens == 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const bool vec = W % 4 == 0 && ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(out)) & (is_fp32 ? 15 : 7)) == 0 &&
                   ((reinterpret_cast<uintptr_t>(mu) | reinterpret_cast<uintptr_t>(state)) & 15) == 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    if (vec) token_shift_vec_kernel<T><<<dim3(tokens, (W / 4 + 255) / 256), 256, 0, s>>>((const T*)h, mu, n_mix, portions, seq_rows, state, (T*)out, tokens, W);
    else token_shift_kernel<T><<<tokens, 256, 0, s>>>((const T*)h, mu, n_mix, portions, seq_rows, state, (T*)out, tokens, W);
  });
  LLMCTL_RETURN_LAST();
}
