// Hyper-connections: S parallel residual streams x_1 .. x_S (fp32, [T, S, W]) around pre-normed sublayers.  A sublayer reads a
// weighted sum of the streams and its output joins every stream, all streams being mixed at the same time:
//
//     u = sum_s a_s x_s;   y = f(layernorm(u));   x_t <- sum_s M[s, t] x_s + b_t y              (M indexed [from, to])
//
//   llmctl_hyper_step  : the update with one sublayer's (M, b) and output y and, from the same pass over the streams, the NEXT
//       sublayer's input layernorm(sum_t a_t x_t) * w + bias in the activation type and, for a router, unrounded in fp32.  a null:
//       plain sum (the model's output norm).  With a list of rows, only those rows' normed sums are formed and nothing is
//       written back (the output norm where logits are wanted).  Without y the streams stay as they are.
//   llmctl_hyper_embed : x_s = scale * table[token] for every stream, and the first sublayer's input.
//
// One CTA per token.  The streams are read and written once, 16 bytes at a time where the width allows; the weighted sum waits in
// shared memory for the row statistics (two passes over it: no cancellation).  Streams, sums, statistics and weights are fp32.
// Reference: none (the reference has no model code).
#include "../common/dtype.cuh"

namespace llmctl {

constexpr int kHyMaxStreams = 16;

struct HyperParams {
  float* x;                   // [T, S, W]
  int S, W;
  const void* y;              // [T, W] sublayer output (row stride ldy), null: no update
  long long ldy;
  const float* mix;           // [S, S]
  const float* out_w;         // [S]
  const float* in_w;          // [S] or null: ones
  const float* w;             // [W] norm weight and bias; null: no norm follows
  const float* b;
  void* out;                  // [rows, W]
  float* out32;               // [rows, W] or null
  const long long* rows;      // null: all tokens, streams written back
  const long long* tokens;    // hyper_embed
  const void* table;
  float scale, eps;
};

// layer norm of the row u (shared memory, each thread reads only the columns it wrote); s: this thread's partial sum of them
template <typename TO, int VEC>
__device__ __forceinline__ void hyper_norm_row(const HyperParams& p, const float* u, float s, long long r, float* red) {
  const int W = p.W;
  const float mean = block_sum(s, red) / static_cast<float>(W);
  float q = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<VEC>(u + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) q += (v[i] - mean) * (v[i] - mean);
  }
  const float rstd = 1.f / sqrtf(block_sum(q, red) / static_cast<float>(W) + p.eps);
  TO* out = static_cast<TO*>(p.out) + r * W;
  float* out32 = p.out32 ? p.out32 + r * W : nullptr;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC], w[VEC], b[VEC];
    load_vec<VEC>(u + c, v);
    load_vec<VEC>(p.w + c, w);
    load_vec<VEC>(p.b + c, b);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = (v[i] - mean) * rstd * w[i] + b[i];
    store_vec<VEC>(out + c, v);
    if (out32) store_vec<VEC>(out32 + c, v);
  }
}

// NS: number of streams (p.S), or kHyMaxStreams for any number up to that
template <typename TY, typename TO, int NS, int VEC>
__global__ void __launch_bounds__(512)
hyper_step_kernel(const HyperParams p) {
  extern __shared__ __align__(16) float hy_u[];          // [W]
  __shared__ float red[32];
  __shared__ float sm[kHyMaxStreams * (kHyMaxStreams + 2)];
  const int W = p.W, S = NS == kHyMaxStreams ? p.S : NS;
  for (int i = threadIdx.x; i < S * (S + 2); i += blockDim.x) {
    float v = 1.f;
    if (i < S * S) v = p.y ? p.mix[i] : 0.f;
    else if (i < S * S + S) v = p.y ? p.out_w[i - S * S] : 0.f;
    else if (p.in_w) v = p.in_w[i - S * S - S];
    sm[i] = v;
  }
  __syncthreads();
  const float* so = sm + S * S;
  const float* si = so + S;
  const long long r = blockIdx.x, t = p.rows ? p.rows[r] : r;
  float* xr = p.x + t * S * W;
  const TY* yr = p.y ? static_cast<const TY*>(p.y) + t * p.ldy : nullptr;
  float sum = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float x[NS][VEC], y[VEC], u[VEC];
#pragma unroll
    for (int s = 0; s < NS; ++s)
      if (s < S) load_vec<VEC>(xr + static_cast<long long>(s) * W + c, x[s]);
    if (yr) load_vec<VEC>(yr + c, y);
#pragma unroll
    for (int i = 0; i < VEC; ++i) u[i] = 0.f;
#pragma unroll
    for (int k = 0; k < NS; ++k)
      if (k < S) {
        float v[VEC];
        if (yr) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[i] = so[k] * y[i];
#pragma unroll
          for (int s = 0; s < NS; ++s)
            if (s < S) {
              const float m = sm[s * S + k];
#pragma unroll
              for (int i = 0; i < VEC; ++i) v[i] = fmaf(m, x[s][i], v[i]);
            }
          if (!p.rows) store_vec<VEC>(xr + static_cast<long long>(k) * W + c, v);
        } else {
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[i] = x[k][i];
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = fmaf(si[k], v[i], u[i]);
      }
    if (p.w) {
      store_vec<VEC>(hy_u + c, u);
#pragma unroll
      for (int i = 0; i < VEC; ++i) sum += u[i];
    }
  }
  if (p.w) hyper_norm_row<TO, VEC>(p, hy_u, sum, r, red);
}

template <typename T, typename TO, int VEC>
__global__ void __launch_bounds__(512)
hyper_embed_kernel(const HyperParams p) {
  extern __shared__ __align__(16) float hy_u[];
  __shared__ float red[32];
  const int W = p.W, S = p.S;
  const long long t = blockIdx.x;
  const T* row = static_cast<const T*>(p.table) + p.tokens[t] * W;
  float total = 0.f;
  for (int s = 0; s < S; ++s) total += p.in_w ? p.in_w[s] : 1.f;
  float sum = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<VEC>(row + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] *= p.scale;
    for (int s = 0; s < S; ++s) store_vec<VEC>(p.x + (t * S + s) * W + c, v);
    if (p.w) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        v[i] *= total;
        sum += v[i];
      }
      store_vec<VEC>(hy_u + c, v);
    }
  }
  if (p.w) hyper_norm_row<TO, VEC>(p, hy_u, sum, t, red);
}

// few rows: wide CTAs (each row's latency counts); many rows: eight CTAs of 256 threads per SM
static int hyper_threads(int rows, int W, int vec) {
  const int want = (W / vec + 31) / 32 * 32, most = rows <= 2 * kNumSMs ? 512 : 256;
  return want < 32 ? 32 : want < most ? want : most;
}

template <typename TY, typename TO, int VEC>
static int launch_hyper_step(const HyperParams& p, int rows, size_t smem, cudaStream_t s) {
  const int threads = hyper_threads(rows, p.W, VEC);
#define LLMCTL_HY_LAUNCH(NS)                                                                                                     \
  do {                                                                                                                           \
    auto kern = hyper_step_kernel<TY, TO, NS, NS == kHyMaxStreams ? 1 : VEC>;                                                                              \
    if (smem > 46 * 1024) LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem))); \
    kern<<<rows, threads, smem, s>>>(p);                                                                                         \
  } while (0)
  switch (p.S) {
    case 1: LLMCTL_HY_LAUNCH(1); break;
    case 2: LLMCTL_HY_LAUNCH(2); break;
    case 3: LLMCTL_HY_LAUNCH(3); break;
    case 4: LLMCTL_HY_LAUNCH(4); break;
    default: if (VEC == 1) LLMCTL_HY_LAUNCH(kHyMaxStreams);      // vec is off for more than four streams
  }
#undef LLMCTL_HY_LAUNCH
  return 0;
}

}  // namespace llmctl

using namespace llmctl;

// x: fp32 [T, S, W]; y: [T, W] (fp32 if y_fp32 else bf16, row stride ldy) or null; mix [S, S], out_w [S], in_w [S] (null: ones); w, b
// [W] or null (no norm); out: [n, W] (fp32 if out_fp32 else bf16); out32: fp32 [n, W] or null; rows: int64 [n] or null (n = T).
LLMCTL_API int llmctl_hyper_step(float* x, int S, const void* y, int y_fp32, long long ldy, const float* mix, const float* out_w,
                                 const float* in_w, const float* w, const float* b, void* out, int out_fp32, float* out32,
                                 const long long* rows, int n, int W, float eps, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(x != nullptr && W > 0 && n >= 0 && S >= 1 && S <= kHyMaxStreams);
  LLMCTL_REQUIRE((!y || (mix && out_w && ldy >= W)) && (!w || (b && out)) && (w || !rows));
  if (n == 0) return 0;
  const HyperParams p{x, S, W, y, ldy, mix, out_w, in_w, w, b, out, out32, rows, nullptr, nullptr, 1.f, eps};
  const size_t smem = sizeof(float) * static_cast<size_t>(W);
  LLMCTL_REQUIRE(smem <= 200 * 1024);
  auto ok = [](const void* q, uintptr_t mask) { return (reinterpret_cast<uintptr_t>(q) & mask) == 0; };
  const bool vec = W % 4 == 0 && S <= 4 && ok(x, 15) && ok(y, y_fp32 ? 15 : 7) && (!y || ldy % 4 == 0) && ok(w, 15) && ok(b, 15) && ok(out, out_fp32 ? 15 : 7) && ok(out32, 15);
  cudaStream_t s = (cudaStream_t)stream;
  int rc = 0;
  LLMCTL_DISPATCH_DTYPE(y_fp32, TY, {
    using TYY = TY;
    LLMCTL_DISPATCH_DTYPE(out_fp32, TO, (rc = vec ? launch_hyper_step<TYY, TO, 4>(p, n, smem, s) : launch_hyper_step<TYY, TO, 1>(p, n, smem, s)));
  });
  if (rc) return rc;
  LLMCTL_RETURN_LAST();
}

// table: [vocab, W] (fp32 if is_fp32 else bf16); x: fp32 [T, S, W]; in_w [S] or null (ones); w, b, out (the table's type), out32 as above.
LLMCTL_API int llmctl_hyper_embed(const long long* tokens, const void* table, int is_fp32, float scale, float* x, int S, const float* in_w,
                                  const float* w, const float* b, void* out, float* out32, int T, int W, float eps, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(x != nullptr && table != nullptr && W > 0 && T >= 0 && S >= 1 && S <= kHyMaxStreams && (!w || (b && out)));
  if (T == 0) return 0;
  const HyperParams p{x, S, W, nullptr, 0, nullptr, nullptr, in_w, w, b, out, out32, nullptr, tokens, table, scale, eps};
  const size_t smem = sizeof(float) * static_cast<size_t>(W);
  LLMCTL_REQUIRE(smem <= 200 * 1024);
  auto ok = [](const void* q, uintptr_t mask) { return (reinterpret_cast<uintptr_t>(q) & mask) == 0; };
  const uintptr_t al = is_fp32 ? 15 : 7;
  const bool vec = W % 4 == 0 && ok(x, 15) && ok(table, al) && ok(w, 15) && ok(b, 15) && ok(out, al) && ok(out32, 15);
  cudaStream_t s = (cudaStream_t)stream;
  LLMCTL_DISPATCH_DTYPE(is_fp32, TT, {
    auto kern = vec ? hyper_embed_kernel<TT, TT, 4> : hyper_embed_kernel<TT, TT, 1>;
    if (smem > 46 * 1024) LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    kern<<<T, hyper_threads(T, W, vec ? 4 : 1), smem, s>>>(p);
  });
  LLMCTL_RETURN_LAST();
}
