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
//   (scan and step are templates in matrix_state.cuh, which retention.cu shares)
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
#include "matrix_state.cuh"

namespace llmctl {

// ---------------------------------------------------------------------------------------------------------------
// prepare
// ---------------------------------------------------------------------------------------------------------------
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

}  // namespace llmctl

using namespace llmctl;

// fp32 numbers of scratch that the prepare and scan entry points need for `tokens` tokens
LLMCTL_API long long llmctl_matrix_scan_work(int tokens, int H, int G, int d, int e, int kind) {
  const long long dp = ms_pad_rows(d), ep = ms_pad_cols(e), T = tokens;
  return T * (2LL * G * dp + H * ep + 4LL * H + (ms_row_decay(kind) ? H * dp : 0));
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
                     norm_w, norm_stride, gate, ldg, gate_kind, eps, out, H, G, d, e, nullptr, nullptr, 0};
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
