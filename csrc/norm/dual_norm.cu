// Residual update and the two pre-norms of a parallel layer (mixer and feed-forward read the same fp32 stream, each through
// its own weighted RMS norm):
//
//     x <- x + (m + f) [+ r]                                 m: mixer output, f: feed-forward output, r: fp32 rows (a stream
//                                                            that joins again before a repeated pass over the layers)
//     out_s = w_s * x / sqrt(mean(x^2) + eps)                s = 0, 1 (one set of statistics: both norms see the same x)
//
// A mixer may be a pair of branches a, b that are normed over the model width before they join:
//
//     m = half_sum * (wa * a / rms(a) + wb * b / rms(b))
//
//   llmctl_residual_dual_norm : all of it in one pass over the rows, one CTA per row.  Rows of up to 8192 numbers whose
//       width is a multiple of 4 stay in registers between the statistics and the outputs (16-byte accesses); other rows
//       are read again.
//   llmctl_embed_sinusoid     : x[t] = scale * table[token[t]] + the sinusoidal position vector (sine at even, cosine at odd
//       columns), in one or two copies.  The angle position * frequency is formed and reduced in fp64, sine and cosine
//       are fp32.
// The stream, sums and weights are fp32; a, b, f and the outputs have the activation type.
// Reference: none (the reference has no model code).
#include "../common/dtype.cuh"

namespace llmctl {

struct DualNormParams {
  const void* a;          // [T, W] mixer output (or first branch), null: none
  const void* b;          // second branch, null: the mixer has one output
  const void* f;          // feed-forward output, null: none
  long long lda, ldb, ldf;
  const float* wa;        // [W] branch weights (with b)
  const float* wb;
  float half_sum;         // factor of the branch sum
  const float* add;       // [T, W] fp32 or null
  float* x;               // [T, W]
  int S;                  // number of outputs, 0 .. 2
  const float* w0;
  const float* w1;
  void* out0;
  void* out1;
  int W;
  float eps;
};

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float dot4(float4 a, float4 b) { return a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w; }

// two block sums at once; red: 64 floats
__device__ __forceinline__ float2 block_sum2(float u, float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
  u = warp_sum(u);
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = u, red[32 + warp] = v;
  __syncthreads();
  return make_float2(warp_sum(lane < nwarp ? red[lane] : 0.f), warp_sum(lane < nwarp ? red[32 + lane] : 0.f));
}

// VPT groups of four columns per thread, held in registers
template <typename T, int VPT, bool PAIR>
__global__ void __launch_bounds__(256)
residual_dual_norm_vec_kernel(const DualNormParams p) {
  __shared__ float red[64];
  const long long t = blockIdx.x;
  const int W = p.W;
  float* xr = p.x + t * W;
  const T* ar = p.a ? static_cast<const T*>(p.a) + t * p.lda : nullptr;
  const T* fr = p.f ? static_cast<const T*>(p.f) + t * p.ldf : nullptr;
  const float* er = p.add ? p.add + t * W : nullptr;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 x[VPT], m[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) << 2;
    x[i] = c < W ? ld4(xr + c) : zero;
    m[i] = (c < W && ar) ? ld4(ar + c) : zero;
  }
  if (PAIR) {
    const T* br = static_cast<const T*>(p.b) + t * p.ldb;
    float4 b[VPT];
    float sa = 0.f, sb = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) << 2;
      b[i] = c < W ? ld4(br + c) : zero;
      sa += dot4(m[i], m[i]);
      sb += dot4(b[i], b[i]);
    }
    const float2 ss = block_sum2(sa, sb, red);
    const float fa = p.half_sum / sqrtf(ss.x / static_cast<float>(W) + p.eps), fb = p.half_sum / sqrtf(ss.y / static_cast<float>(W) + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) << 2;
      if (c < W) {
        const float4 wa = ld4(p.wa + c), wb = ld4(p.wb + c);
        m[i].x = m[i].x * fa * wa.x + b[i].x * fb * wb.x;
        m[i].y = m[i].y * fa * wa.y + b[i].y * fb * wb.y;
        m[i].z = m[i].z * fa * wa.z + b[i].z * fb * wb.z;
        m[i].w = m[i].w * fa * wa.w + b[i].w * fb * wb.w;
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) << 2;
    if (c < W) {
      if (fr) {
        const float4 f = ld4(fr + c);
        m[i].x += f.x, m[i].y += f.y, m[i].z += f.z, m[i].w += f.w;
      }
      x[i].x += m[i].x, x[i].y += m[i].y, x[i].z += m[i].z, x[i].w += m[i].w;
      if (er) {
        const float4 e = ld4(er + c);
        x[i].x += e.x, x[i].y += e.y, x[i].z += e.z, x[i].w += e.w;
      }
      if (ar || fr || er) st4(xr + c, x[i]);
      ss += dot4(x[i], x[i]);
    }
  }
  if (p.S == 0) return;
  const float r = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(W) + p.eps);
  T* o0 = static_cast<T*>(p.out0) + t * W;
  T* o1 = p.S > 1 ? static_cast<T*>(p.out1) + t * W : nullptr;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) << 2;
    if (c < W) {
      const float4 n = make_float4(x[i].x * r, x[i].y * r, x[i].z * r, x[i].w * r);
      const float4 w = ld4(p.w0 + c);
      st4(o0 + c, make_float4(n.x * w.x, n.y * w.y, n.z * w.z, n.w * w.w));
      if (o1) {
        const float4 u = ld4(p.w1 + c);
        st4(o1 + c, make_float4(n.x * u.x, n.y * u.y, n.z * u.z, n.w * u.w));
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
residual_dual_norm_kernel(const DualNormParams p) {
  __shared__ float red[64];
  const long long t = blockIdx.x;
  const int W = p.W;
  float* xr = p.x + t * W;
  const T* ar = p.a ? static_cast<const T*>(p.a) + t * p.lda : nullptr;
  const T* br = p.b ? static_cast<const T*>(p.b) + t * p.ldb : nullptr;
  const T* fr = p.f ? static_cast<const T*>(p.f) + t * p.ldf : nullptr;
  const float* er = p.add ? p.add + t * W : nullptr;
  float fa = 1.f, fb = 0.f;
  if (br) {
    float sa = 0.f, sb = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float a = to_f32(ar[c]), b = to_f32(br[c]);
      sa += a * a;
      sb += b * b;
    }
    const float2 s2 = block_sum2(sa, sb, red);
    fa = p.half_sum / sqrtf(s2.x / static_cast<float>(W) + p.eps);
    fb = p.half_sum / sqrtf(s2.y / static_cast<float>(W) + p.eps);
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {       // a thread reads again only what it wrote itself
    float m = ar ? to_f32(ar[c]) : 0.f;
    if (br) m = m * fa * p.wa[c] + to_f32(br[c]) * fb * p.wb[c];
    if (fr) m += to_f32(fr[c]);
    float v = xr[c] + m;
    if (er) v += er[c];
    if (ar || fr || er) xr[c] = v;
    ss += v * v;
  }
  if (p.S == 0) return;
  const float r = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(W) + p.eps);
  T* o0 = static_cast<T*>(p.out0) + t * W;
  T* o1 = p.S > 1 ? static_cast<T*>(p.out1) + t * W : nullptr;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float n = xr[c] * r;
    o0[c] = from_f32<T>(n * p.w0[c]);
    if (o1) o1[c] = from_f32<T>(n * p.w1[c]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
embed_sinusoid_kernel(const long long* __restrict__ tokens, const int* __restrict__ positions, const T* __restrict__ table, float scale,
                      const double* __restrict__ freq, float* __restrict__ x, float* __restrict__ copy, int W) {
  constexpr double kTwoPi = 6.283185307179586476925286766559;
  const long long t = blockIdx.x;
  const T* row = table + tokens[t] * W;
  const double pos = static_cast<double>(positions[t]);
  for (int i = threadIdx.x; 2 * i < W; i += blockDim.x) {
    double a = pos * freq[i];
    a -= kTwoPi * rint(a / kTwoPi);
    float s, c;
    sincosf(static_cast<float>(a), &s, &c);
    const long long o = t * W + 2 * i;
    const float v = to_f32(row[2 * i]) * scale + s;
    x[o] = v;
    if (copy) copy[o] = v;
    if (2 * i + 1 < W) {
      const float u = to_f32(row[2 * i + 1]) * scale + c;
      x[o + 1] = u;
      if (copy) copy[o + 1] = u;
    }
  }
}

template <typename T, int VPT>
static void launch_dual_norm_vec(const DualNormParams& p, int rows, int threads, cudaStream_t s) {
  if (p.b) residual_dual_norm_vec_kernel<T, VPT, true><<<rows, threads, 0, s>>>(p);
  else residual_dual_norm_vec_kernel<T, VPT, false><<<rows, threads, 0, s>>>(p);
}

template <typename T>
static void launch_dual_norm(const DualNormParams& p, int rows, bool vec, cudaStream_t s) {
  const int groups = p.W >> 2;
  if (!vec || groups > 8 * 256) {
    residual_dual_norm_kernel<T><<<rows, 256, 0, s>>>(p);
    return;
  }
  const int per = groups <= 256 ? 1 : groups <= 512 ? 2 : groups <= 1024 ? 4 : 8;
  const int threads = ((groups + per - 1) / per + 31) / 32 * 32;
  if (per == 1) launch_dual_norm_vec<T, 1>(p, rows, threads, s);
  else if (per == 2) launch_dual_norm_vec<T, 2>(p, rows, threads, s);
  else if (per == 4) launch_dual_norm_vec<T, 4>(p, rows, threads, s);
  else launch_dual_norm_vec<T, 8>(p, rows, threads, s);
}

}  // namespace llmctl

using namespace llmctl;

// a, b, f: [rows, W] in the activation type (row strides lda, ldb, ldf) or null; b needs a, wa and wb; add: fp32 [rows, W] or
// null; x: fp32 [rows, W] in place; S outputs of [rows, W] with fp32 weights.
LLMCTL_API int llmctl_residual_dual_norm(const void* a, long long lda, const void* b, long long ldb, const float* wa, const float* wb,
                                         float half_sum, const void* f, long long ldf, const float* add, float* x, int S,
                                         const float* w0, void* out0, const float* w1, void* out1, int rows, int W, float eps,
                                         int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(W > 0 && rows >= 0 && S >= 0 && S <= 2 && x != nullptr);
  LLMCTL_REQUIRE((S < 1 || (w0 && out0)) && (S < 2 || (w1 && out1)) && (!b || (a && wa && wb)));
  LLMCTL_REQUIRE((!a || lda >= W) && (!b || ldb >= W) && (!f || ldf >= W));
  if (rows == 0) return 0;
  DualNormParams p{a, b, f, lda, ldb, ldf, wa, wb, half_sum, add, x, S, w0, w1, out0, out1, W, eps};
  const uintptr_t al = is_fp32 ? 15 : 7;
  auto ok = [&](const void* q, long long ld, uintptr_t mask) { return q == nullptr || ((reinterpret_cast<uintptr_t>(q) & mask) == 0 && ld % 4 == 0); };
  const bool vec = W % 4 == 0 && ok(a, lda, al) && ok(b, ldb, al) && ok(f, ldf, al) && ok(add, 4, 15) && ok(x, 4, 15) && ok(wa, 4, 15) &&
                   ok(wb, 4, 15) && ok(w0, 4, 15) && ok(w1, 4, 15) && ok(out0, 4, al) && ok(out1, 4, al);
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (launch_dual_norm<T>(p, rows, vec, (cudaStream_t)stream)));
  LLMCTL_RETURN_LAST();
}

// freq: fp64 [(W + 1) / 2]; x and copy (or null): fp32 [rows, W].
LLMCTL_API int llmctl_embed_sinusoid(const long long* tokens, const int* positions, const void* table, int is_fp32, float scale,
                                     const double* freq, float* x, float* copy, int rows, int W, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(W > 0 && rows >= 0);
  if (rows == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (embed_sinusoid_kernel<T><<<rows, 256, 0, (cudaStream_t)stream>>>(tokens, positions, (const T*)table, scale,
                                                                                                      freq, x, copy, W)));
  LLMCTL_RETURN_LAST();
}
