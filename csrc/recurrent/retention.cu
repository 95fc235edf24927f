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
