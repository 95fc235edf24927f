// Post-processing of a packed query / key / value projection and append to a paged cache whose token rows hold the keys of all
// key/value heads and then their values, for bf16 or fp32 activations.
//
//   llmctl_window_qkv_write : per token, from the packed projection [q | k | v]: + bias, RMS norm over the whole q
//       and the whole k projection (per-coordinate weights), rotation of the first `rot` numbers of every head at the token's
//       position (pairs of neighbours (2i, 2i + 1), or pairs (i, i + rot/2) when `rot_half`), value mixing
//       v <- (1-lam) v + lam v_first with the values an earlier layer computed for the same token; q leaves in fp32, k and v
//       go to the token's cache row (pages of bs token rows and PS further rows).
//
// One CTA per token: the projection passes through shared memory once, sines and cosines are evaluated once per token and
// pair and shared by the heads, rows whose sizes and addresses allow it move in groups of four numbers.  Sums, norms,
// angles and rotations are fp32.
// Reference: none (the reference has no attention code; reference llmctl/serve/server.py:199-204 calls HF).
#include "../common/dtype.cuh"

namespace llmctl {

struct QkvWriteParams {
  const void* qkv;
  long long ld;
  const void* bias;           // [Nq + Nk + Nv] or null; fp32 if bias_fp32, else the activation type
  int bias_fp32;
  const float* qn_w;          // [Nq] / [Nk] or null: no norm
  const float* kn_w;
  int H, G, d, e, rot, rot_half;
  const float* freq;          // [rot / 2]
  float mult, eps;
  const int* positions;
  const long long* slots;
  float* q_out;               // [T, Nq]
  void* cache;
  int bs, PS;
  void* v_first;              // [T, Nv]
  int v_mode;
  const float* lam;
};

template <typename T, int VEC>
__device__ __forceinline__ void add_bias(const QkvWriteParams& p, int c, float (&v)[VEC]) {
  if (!p.bias) return;
  float b[VEC];
  if (p.bias_fp32) load_vec<VEC>(static_cast<const float*>(p.bias) + c, b);
  else load_vec<VEC>(static_cast<const T*>(p.bias) + c, b);
#pragma unroll
  for (int i = 0; i < VEC; ++i) v[i] += b[i];
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
window_qkv_write_kernel(const QkvWriteParams p) {
  extern __shared__ __align__(16) float buf[];      // [Nq + Nk] projections, then [rot / 2] (cos, sin)
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int H = p.H, G = p.G, d = p.d, Nq = H * d, Nk = G * d, Nv = G * p.e, Wc = Nk + Nv, rot = p.rot, half = rot >> 1;
  const T* row = static_cast<const T*>(p.qkv) + t * p.ld;
  float2* cs = reinterpret_cast<float2*>(buf + ((Nq + Nk + 3) & ~3));
  const int pos = p.positions[t];
  const long long slot = p.slots[t];
  float ssq = 0.f, ssk = 0.f;
  for (int c = threadIdx.x * VEC; c < Nq + Nk; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<VEC>(row + c, v);
    add_bias<T, VEC>(p, c, v);
    store_vec<VEC>(buf + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) (c < Nq ? ssq : ssk) += v[i] * v[i];
  }
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(static_cast<float>(pos) * p.freq[i], &s, &c);
    cs[i] = make_float2(c * p.mult, s * p.mult);
  }
  ssq = block_sum(ssq, red);                        // its barriers also publish buf and cs
  ssk = block_sum(ssk, red);
  const float rq = p.qn_w ? 1.f / sqrtf(ssq / static_cast<float>(Nq) + p.eps) : 1.f;
  const float rk = p.kn_w ? 1.f / sqrtf(ssk / static_cast<float>(Nk) + p.eps) : 1.f;
  T* crow = slot >= 0 ? static_cast<T*>(p.cache) + ((slot / p.bs) * (p.bs + p.PS) + slot % p.bs) * Wc : nullptr;
  for (int c = threadIdx.x * VEC; c < Nq + Nk; c += blockDim.x * VEC) {
    const bool isq = c < Nq;
    if (!isq && !crow) break;
    const int cc = isq ? c : c - Nq, d0 = cc % d;
    const float* src = buf + c - d0;                // the head's numbers
    const float* w = isq ? p.qn_w : p.kn_w;
    const float r = isq ? rq : rk;
    if (w) w += cc - d0;
    auto normed = [&](int k) { return w ? src[k] * r * w[k] : src[k]; };
    float out[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int dd = d0 + i;
      float v = normed(dd);
      if (dd < rot) {
        const bool second = p.rot_half ? dd >= half : (dd & 1);
        const int pair = p.rot_half ? (second ? dd - half : dd) : dd >> 1;
        const int other = p.rot_half ? (second ? dd - half : dd + half) : dd ^ 1;
        const float2 a = cs[pair];
        const float u = normed(other);
        v = second ? v * a.x + u * a.y : v * a.x - u * a.y;
      }
      out[i] = v;
    }
    if (isq) store_vec<VEC>(p.q_out + t * Nq + cc, out);
    else store_vec<VEC>(crow + cc, out);
  }
  const float l = (p.v_mode == 2) ? p.lam[0] : 0.f;
  for (int c = threadIdx.x * VEC; c < Nv; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<VEC>(row + Nq + Nk + c, v);
    add_bias<T, VEC>(p, Nq + Nk + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = to_f32(from_f32<T>(v[i]));      // the projection's output in the activation type
    T* vf = p.v_mode ? static_cast<T*>(p.v_first) + t * Nv + c : nullptr;
    if (p.v_mode == 1) store_vec<VEC>(vf, v);
    if (p.v_mode == 2) {
      float f[VEC];
      load_vec<VEC>(vf, f);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = (1.f - l) * v[i] + l * f[i];
    }
    if (crow) store_vec<VEC>(crow + Nk + c, v);
  }
}

}  // namespace llmctl

using namespace llmctl;

LLMCTL_API int llmctl_window_qkv_write(const void* qkv, long long ld, const void* bias, int bias_fp32, const float* qn_w, const float* kn_w,
                                       int H, int G, int d, int e, int rot, int rot_half, const float* freq, float mult, float eps,
                                       const int* positions, const long long* slots, float* q_out, void* cache, int bs, int PS,
                                       void* v_first, int v_mode, const float* lam, int tokens, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(H > 0 && G > 0 && H % G == 0 && d > 0 && e > 0 && rot >= 0 && rot <= d && rot % 2 == 0 && bs > 0 && PS >= 0);
  LLMCTL_REQUIRE(v_mode == 0 || (v_first != nullptr && (v_mode == 1 || lam != nullptr)));
  LLMCTL_REQUIRE(rot == 0 || freq != nullptr);
  if (tokens == 0) return 0;
  const size_t smem = (static_cast<size_t>(H + G) * d + 4 + rot) * sizeof(float);
  LLMCTL_REQUIRE(smem <= 200 * 1024);
  cudaStream_t s = (cudaStream_t)stream;
  const QkvWriteParams p{qkv, ld, bias, bias_fp32, qn_w, kn_w, H, G, d, e, rot, rot_half, freq, mult, eps, positions, slots, q_out, cache, bs, PS,
                         v_first, v_mode, lam};
  const uintptr_t al = is_fp32 ? 15 : 7;
  auto ok = [](const void* q, uintptr_t mask) { return (reinterpret_cast<uintptr_t>(q) & mask) == 0; };
  const bool vec = d % 4 == 0 && e % 4 == 0 && ld % 4 == 0 && ok(qkv, al) && ok(cache, al) && ok(v_first, al) && ok(q_out, 15) &&
                   ok(bias, bias_fp32 ? 15 : al);
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    auto kern = vec ? window_qkv_write_kernel<T, 4> : window_qkv_write_kernel<T, 1>;
    if (smem > 46 * 1024) LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    kern<<<tokens, 256, smem, s>>>(p);
  });
  LLMCTL_RETURN_LAST();
}
