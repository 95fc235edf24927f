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
//   llmctl_matrix_scan : the serial part.  A CTA owns (portion, head, 16 or 32 value columns).  LPC lanes share one or two
//       columns, each with d / LPC rows of them in registers; a token costs one pass over them (decay, S^T k and S^T q together: the
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
constexpr int kMsCols = 32;         // most value columns per CTA of the scan
constexpr int kMsNarrow = 148;      // up to this many CTAs of the wide scan: the narrow one runs
constexpr int kMsWalk = 64;         // most consecutive tokens a warp of the delta prepare kernel walks

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
  int walk;                   // tokens per walk
  MsWork w;
};

// raw input of channel c at token row src (< t0: from the state slot's rows, zeros before the sequence)
template <typename T>
__device__ __forceinline__ float ms_raw(const T* x, long long ldx, long long src, int t0, const float* st, int keep, int C, int c) {
  if (src >= t0) return to_f32(x[src * ldx + c]);
  return st ? st[static_cast<long long>(keep - (t0 - src)) * C + c] : 0.f;
}

// silu of a short convolution: bf16 inputs carry 8 bits, so the hardware's exponential and reciprocal are exact enough there
template <typename T>
__device__ __forceinline__ float ms_conv_act(float x) {
  if (sizeof(T) == 2) return __fdividef(x, 1.f + __expf(-fmaxf(x, -80.f)));
  return ms_silu(x);
}

// Short convolution of one channel along consecutive tokens.  SHORT (up to four taps): weights and history in registers;
// otherwise every tap is read again.
template <typename T, bool SHORT>
struct ConvWalk {
  float w[SHORT ? 4 : 1], h[SHORT ? 3 : 1];
  __device__ __forceinline__ void weights(const float* conv_w, int taps, int c) {
    if (!SHORT) return;
    if (taps == 4) {
      const float4 v = *reinterpret_cast<const float4*>(conv_w + static_cast<long long>(c) * 4);
      w[0] = v.x, w[SHORT ? 1 : 0] = v.y, w[SHORT ? 2 : 0] = v.z, w[SHORT ? 3 : 0] = v.w;
      return;
    }
#pragma unroll
    for (int j = 0; j < (SHORT ? 4 : 0); ++j) {
      const int src = taps - 4 + j;                   // w[3] is the current token's weight
      w[j] = src >= 0 ? conv_w[static_cast<long long>(c) * taps + src] : 0.f;
    }
  }
  __device__ __forceinline__ void history(const T* x, long long ldx, long long t, int t0, const float* st, int taps, int C, int c) {
#pragma unroll
    for (int j = 0; j < (SHORT ? 3 : 0); ++j) {
      const int back = 3 - j;
      h[j] = back <= taps - 1 ? ms_raw(x, ldx, t - back, t0, st, taps - 1, C, c) : 0.f;
    }
  }
  // cur: the channel's raw input of token t
  __device__ __forceinline__ float step(float cur, const T* x, long long ldx, long long t, int t0, const float* st, const float* conv_w,
                                        int taps, int C, int c) {
    float a;
    if (SHORT) {
      a = w[0] * h[0] + w[SHORT ? 1 : 0] * h[SHORT ? 1 : 0] + w[SHORT ? 2 : 0] * h[SHORT ? 2 : 0] + w[SHORT ? 3 : 0] * cur;
      h[0] = h[SHORT ? 1 : 0];
      h[SHORT ? 1 : 0] = h[SHORT ? 2 : 0];
      h[SHORT ? 2 : 0] = cur;
    } else {
      a = conv_w[static_cast<long long>(c) * taps + taps - 1] * cur;
      for (int j = 0; j < taps - 1; ++j)
        a += conv_w[static_cast<long long>(c) * taps + j] * ms_raw(x, ldx, t - (taps - 1 - j), t0, st, taps - 1, C, c);
    }
    return ms_conv_act<T>(a);
  }
};

// A warp is one unit: units 0 .. G-1 are the query and key of a key/value head, then blocks of 128 padded value columns,
// then (kind 1) blocks of 128 padded decay columns.  blockIdx.x: a walk of p.walk tokens; the next token's raw inputs are
// asked for before the current one's are used.
template <typename T, int NI, bool SHORT>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaPrepParams p) {
  const int lane = threadIdx.x & 31;
  const int H = p.H, G = p.G, d = p.d, e = p.e, taps = p.taps, keep = taps - 1;
  const int dp = ms_pad_rows(d), ep = ms_pad_cols(e), rep = H / G, C = 2 * G * d + H * e;
  const int nv = (H * ep + 127) / 128, nd = p.kind == 1 ? (H * dp + 127) / 128 : 0;
  int unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (unit >= G + nv + nd) return;
  const int tb = blockIdx.x * p.walk, te = min(tb + p.walk, p.T);
  const T none = from_f32<T>(0.f);
  int t0 = 0, t_end = -1;
  const float* st = nullptr;
  auto enter = [&](int t) {               // true when token t opens a portion (or the walk): histories are stale
    if (t < t_end) return false;
    const int* pt = p.portions + 4 * p.seq_rows[t];
    t0 = pt[0];
    t_end = t0 + pt[1];
    st = (pt[2] > 0 && pt[3] >= 0) ? p.conv_state + static_cast<long long>(pt[3]) * keep * C : nullptr;
    return true;
  };
  if (unit < G) {
    const int g = unit;
    const T* x = static_cast<const T*>(p.x);
    ConvWalk<T, SHORT> cq[NI], ck[NI];
    T nq[NI], nk[NI];
    const T* row = x + tb * p.ldx + g * d + lane;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = lane + 32 * i;
      nq[i] = nk[i] = none;
      if (c < d) {
        cq[i].weights(p.conv_w, taps, g * d + c);
        ck[i].weights(p.conv_w, taps, (G + g) * d + c);
        nq[i] = row[32 * i];
        nk[i] = row[32 * i + G * d];
      }
    }
    const float qs = rsqrtf(static_cast<float>(d));
#pragma unroll 1
    for (int t = tb; t < te; ++t) {
      float q[NI], k[NI], sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) q[i] = to_f32(nq[i]), k[i] = to_f32(nk[i]);
      row += p.ldx;
      if (t + 1 < te) {
#pragma unroll
        for (int i = 0; i < NI; ++i)
          if (lane + 32 * i < d) {
            nq[i] = row[32 * i];
            nk[i] = row[32 * i + G * d];
          }
      }
      if (enter(t) && SHORT) {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int c = lane + 32 * i;
          if (c < d) {
            cq[i].history(x, p.ldx, t, t0, st, taps, C, g * d + c);
            ck[i].history(x, p.ldx, t, t0, st, taps, C, (G + g) * d + c);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int c = lane + 32 * i;
        if (c < d) {
          q[i] = cq[i].step(q[i], x, p.ldx, t, t0, st, p.conv_w, taps, C, g * d + c);
          k[i] = ck[i].step(k[i], x, p.ldx, t, t0, st, p.conv_w, taps, C, (G + g) * d + c);
        }
        sq += q[i] * q[i];
        sk += k[i] * k[i];
        qk += q[i] * k[i];
      }
      const float fq = qs / sqrtf(warp_sum(sq) + 1e-6f), fk = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
      qk = warp_sum(qk) * fq * fk;
      float* wq = p.w.q + (static_cast<long long>(t) * G + g) * dp + lane;
      float* wk = p.w.k + (static_cast<long long>(t) * G + g) * dp + lane;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        wq[32 * i] = q[i] * fq;
        wk[32 * i] = k[i] * fk;
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
  const bool value = unit < nv;
  if (!value) unit -= nv;
  const int width = value ? ep : dp, real = value ? e : d;
  const T* x = static_cast<const T*>(value ? p.x : p.z);
  const long long ldx = value ? p.ldx : p.ldz;
  float* out = (value ? p.w.v : p.w.dm) + static_cast<long long>(tb) * H * width + unit * 128 + lane;
  ConvWalk<T, SHORT> cv[4];
  int ch[4];
  float sp[4], bias[4];
  T nx[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int col = unit * 128 + lane + 32 * i, h = col / width, c = col % width;
    const bool ok = h < H && c < real;
    ch[i] = ok ? (value ? 2 * G * d : 0) + h * real + c : -1;
    sp[i] = bias[i] = 0.f;
    nx[i] = none;
    if (ok) {
      nx[i] = x[tb * ldx + ch[i]];
      if (value) {
        cv[i].weights(p.conv_w, taps, ch[i]);
      } else {
        sp[i] = p.speed[h];
        bias[i] = p.dt_bias[ch[i]];
      }
    }
  }
#pragma unroll 1
  for (int t = tb; t < te; ++t, out += H * width) {
    float v[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = to_f32(nx[i]);
    if (t + 1 < te) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (ch[i] >= 0) nx[i] = x[(t + 1) * ldx + ch[i]];
    }
    if (value) {
      if (enter(t) && SHORT) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (ch[i] >= 0) cv[i].history(x, ldx, t, t0, st, taps, C, ch[i]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (ch[i] >= 0) v[i] = cv[i].step(v[i], x, ldx, t, t0, st, p.conv_w, taps, C, ch[i]);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (ch[i] >= 0) v[i] = expm1f(-sp[i] * ms_softplus(v[i] + bias[i]));
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (unit * 128 + lane + 32 * i < H * width) out[32 * i] = v[i];
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

// A token's prepared numbers as a lane holds them.
template <int NP, int CPL, int KIND>
struct ScanToken {
  f32x2 k[NP], q[NP], d[KIND == 0 ? 1 : NP];
  float4 sc;
  float v[CPL];
};

// KIND 0: delta rule, decay per head; 1: delta rule, decay per key row; 2: outer products with a bonus.
// A lane owns columns c0 .. c0 + CPL - 1 and the rows (i LPC + sub) 4 .. + 3, i < RPT / 4; the CTA 16 CPL columns.
template <int RPT, int LPC, int CPL, int KIND>
__global__ void __launch_bounds__(LPC * 16)
matrix_scan_kernel(const MatrixScanParams p) {
  constexpr int TC = kMsTC, DP = RPT * LPC, NG = 32 / LPC, NT = LPC * 16, NP = RPT / 2, COLS = 16 * CPL;
  constexpr int NROW = KIND == 0 ? 2 : 3, STAGE = TC * (DP * NROW + COLS + 4);
  constexpr bool AHEAD = RPT <= 16;          // the next token's numbers are fetched while this one's sums meet
  typedef ScanToken<NP, CPL, KIND> Tok;
  extern __shared__ __align__(16) float ms_smem[];
  const int H = p.H, d = p.d, e = p.e;
  const int* pt = p.portions + blockIdx.x * 4;
  const int t0 = pt[0], n = pt[1], pos0 = pt[2], slot = pt[3];
  if (n <= 0) return;
  const int h = blockIdx.y, kvh = h / (H / p.G), ep = ms_pad_cols(e), cb = blockIdx.z * COLS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = lane % LPC;
  const int cl = (warp * NG + lane / LPC) * CPL;             // first of this lane's columns within the CTA's
  float* so = ms_smem + 2 * STAGE;                           // [2][TC][COLS] outputs of the chunk

  f32x2 S[CPL][NP];
  float* st = slot >= 0 ? p.state + ((static_cast<long long>(slot) * H + h) * d) * e : nullptr;
#pragma unroll
  for (int c = 0; c < CPL; ++c)
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
    float* sv = sk + TC * DP * NROW;
    float* ss = sv + TC * COLS;
    const int cnt = min(TC, n - c0);
    const long long tb = t0 + c0;
    for (int i = tid; i < cnt * (DP / 4); i += NT) {
      const int tok = i / (DP / 4), c = i % (DP / 4) * 4;
      const long long src = ((tb + tok) * p.G + kvh) * DP + c;
      cp_async_16(sk + tok * DP + c, p.w.k + src);
      cp_async_16(sq + tok * DP + c, p.w.q + src);
      if (KIND != 0) cp_async_16(sd + tok * DP + c, p.w.dm + ((tb + tok) * H + h) * DP + c);
    }
    constexpr int VC = COLS / 4;
    for (int i = tid; i < cnt * (VC + 1); i += NT) {
      const int tok = i / (VC + 1), c = i % (VC + 1);
      if (c < VC) cp_async_16(sv + tok * COLS + c * 4, p.w.v + ((tb + tok) * H + h) * ep + cb + c * 4);
      else cp_async_16(ss + tok * 4, p.w.sc + ((tb + tok) * H + h) * 4);
    }
  };
  auto flush = [&](int c0, int buf) {                        // the chunk's outputs, neighbouring columns of a token together
    const int cnt = min(TC, n - c0);
    for (int i = tid; i < cnt * COLS; i += NT) {
      const int tok = i / COLS, c = i % COLS;
      if (cb + c < e) p.out[(static_cast<long long>(t0 + c0 + tok) * H + h) * e + cb + c] = so[(buf * TC + tok) * COLS + c];
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
    const float* sv = ms_smem + buf * STAGE + TC * DP * NROW + cl;
    const float* ss = ms_smem + buf * STAGE + TC * DP * NROW + TC * COLS;
    float* od = so + buf * TC * COLS + cl;
    const int cnt = min(TC, n - c0);

    auto fetch = [&](Tok& w, int tok) {
      w.sc = *reinterpret_cast<const float4*>(ss + tok * 4);
#pragma unroll
      for (int c = 0; c < CPL; ++c) w.v[c] = sv[tok * COLS + c];
#pragma unroll
      for (int i = 0; i < NP; i += 2) {
        ld_pairs(sk + tok * DP + i * 2 * LPC, w.k[i], w.k[i + 1]);
        ld_pairs(sq + tok * DP + i * 2 * LPC, w.q[i], w.q[i + 1]);
        if (KIND != 0) ld_pairs(sd + tok * DP + i * 2 * LPC, w.d[KIND == 0 ? 0 : i], w.d[KIND == 0 ? 0 : i + 1]);
      }
    };
    auto step = [&](const Tok& w, Tok& next, int tok) {
      f32x2 ka[CPL][2], qa[CPL][2];
      const f32x2 dh = pk(w.sc.z, w.sc.z);
#pragma unroll
      for (int c = 0; c < CPL; ++c) ka[c][0] = ka[c][1] = qa[c][0] = qa[c][1] = 0ull;
#pragma unroll
      for (int i = 0; i < NP; ++i)
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          if (KIND == 2) qa[c][i & 1] = fma2(w.q[i], S[c][i], qa[c][i & 1]);       // the read-out precedes this token's write
          S[c][i] = fma2(KIND == 0 ? dh : w.d[KIND == 0 ? 0 : i], S[c][i], S[c][i]);
          if (KIND != 2) ka[c][i & 1] = fma2(w.k[i], S[c][i], ka[c][i & 1]);
        }
      float u[CPL], o[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        u[c] = w.v[c];
        if (KIND != 2) {
          const float2 x = upk(ka[c][0]), y = upk(ka[c][1]);
          o[c] = (x.x + y.x) + (x.y + y.y);
        }
      }
      if (KIND != 2) {                       // the read-out's products fill the waits of these shuffles
#pragma unroll
        for (int off = LPC / 2; off > 0; off >>= 1)
#pragma unroll
          for (int c = 0; c < CPL; ++c) o[c] += __shfl_xor_sync(0xffffffffu, o[c], off);
#pragma unroll
        for (int i = 0; i < NP; ++i)
#pragma unroll
          for (int c = 0; c < CPL; ++c) qa[c][i & 1] = fma2(w.q[i], S[c][i], qa[c][i & 1]);
#pragma unroll
        for (int c = 0; c < CPL; ++c) u[c] = w.sc.x * (w.v[c] - o[c]);
      }
      if (AHEAD) fetch(next, min(tok + 1, TC - 1));
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const f32x2 u2 = pk(u[c], u[c]);
#pragma unroll
        for (int i = 0; i < NP; ++i) S[c][i] = fma2(w.k[i], u2, S[c][i]);
        const float2 x = upk(qa[c][0]), y = upk(qa[c][1]);
        o[c] = (x.x + y.x) + (x.y + y.y);
      }
#pragma unroll
      for (int off = LPC / 2; off > 0; off >>= 1)
#pragma unroll
        for (int c = 0; c < CPL; ++c) o[c] += __shfl_xor_sync(0xffffffffu, o[c], off);
      if (sub == 0) {
#pragma unroll
        for (int c = 0; c < CPL; ++c) od[tok * COLS + c] = o[c] + w.sc.y * u[c];
      }
    };
    Tok wa, wb;
    if (AHEAD) {
      fetch(wa, 0);
      for (int tok = 0; tok < cnt; tok += 2) {
        step(wa, wb, tok);
        if (tok + 1 < cnt) step(wb, wa, tok + 1);
      }
    } else {
#pragma unroll 1
      for (int tok = 0; tok < cnt; ++tok) {
        fetch(wa, tok);
        step(wa, wa, tok);
      }
    }
  }
  __syncthreads();
  flush((n - 1) / TC * TC, buf ^ 1);
  if (!st) return;
#pragma unroll
  for (int c = 0; c < CPL; ++c)
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

template <typename T, int NI>
static void launch_delta_prepare(const DeltaPrepParams& p, dim3 grid, cudaStream_t s) {
  if (p.taps <= 4) delta_prepare_kernel<T, NI, true><<<grid, 256, 0, s>>>(p);
  else delta_prepare_kernel<T, NI, false><<<grid, 256, 0, s>>>(p);
}

template <int RPT, int LPC, int CPL, int KIND>
static int launch_matrix_scan_cols(const MatrixScanParams& p, int nportions, cudaStream_t s) {
  constexpr int DP = RPT * LPC, COLS = 16 * CPL;
  const size_t smem = sizeof(float) * (2 * kMsTC * (static_cast<size_t>(DP) * (KIND == 0 ? 2 : 3) + COLS + 4) + 2 * kMsTC * COLS);
  auto kern = matrix_scan_kernel<RPT, LPC, CPL, KIND>;
  if (smem > 46 * 1024) LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kern<<<dim3(nportions, p.H, (p.e + COLS - 1) / COLS), LPC * 16, smem, s>>>(p);
  return 0;
}

// Two columns per lane share the loads of a token's vectors; with few CTAs a token's latency counts instead, and one
// column per lane halves its work.
template <int RPT, int LPC, int KIND>
static int launch_matrix_scan(const MatrixScanParams& p, int nportions, cudaStream_t s) {
  const long long ctas = static_cast<long long>(nportions) * p.H * (ms_pad_cols(p.e) / kMsCols);
  return ctas <= kMsNarrow ? launch_matrix_scan_cols<RPT, LPC, 1, KIND>(p, nportions, s)
                           : launch_matrix_scan_cols<RPT, LPC, 2, KIND>(p, nportions, s);
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
  LLMCTL_REQUIRE(smem <= 46 * 1024);
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
  LLMCTL_REQUIRE((reinterpret_cast<uintptr_t>(work) & 15) == 0 && (reinterpret_cast<uintptr_t>(conv_w) & 15) == 0);
  LLMCTL_REQUIRE(taps == 1 || conv_state != nullptr);
  if (tokens == 0) return 0;
  DeltaPrepParams p{x, ldx, conv_w, conv_state, z, ldz, dt_bias, speed, b, ldb, portions, seq_rows, tokens, H, G, d, e, taps, kind, kMsWalk,
                    ms_work(work, tokens, H, G, d, e, kind)};
  const int dp = ms_pad_rows(d), ep = ms_pad_cols(e);
  const int units = G + (H * ep + 127) / 128 + (kind == 1 ? (H * dp + 127) / 128 : 0);
  // long walks load weights and histories less often; short ones keep every SM busy
  while (p.walk > 16 && ((tokens + p.walk - 1) / p.walk) * ((units + 7) / 8) < 2 * kNumSMs) p.walk /= 2;
  const dim3 grid((tokens + p.walk - 1) / p.walk, (units + 7) / 8);
  cudaStream_t s = (cudaStream_t)stream;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    if (dp == 32) launch_delta_prepare<T, 1>(p, grid, s);
    else if (dp == 64) launch_delta_prepare<T, 2>(p, grid, s);
    else if (dp == 128) launch_delta_prepare<T, 4>(p, grid, s);
    else launch_delta_prepare<T, 8>(p, grid, s);
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
