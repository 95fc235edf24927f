// Elementwise activations of the feed-forward layers, for bf16 or fp32 activations, evaluated in fp32:
//
//   xIELU        : z > 0 :  a_pos * z^2 + z / 2          a_pos = softplus(p)
//                  z <= 0:  a_neg * (exp(z) - 1 - z) + z / 2,   a_neg = 1/2 + softplus(q)
//                  (the caller passes a_pos and a_neg; they depend on two learned numbers only)
//   gated SiLU   : out = silu(gate) * up on a packed [rows, 2F] activation (gate first) of either type
//                  (csrc/swiglu/swiglu.cu is the bf16-only training kernel with a backward).
//   squared ReLU : max(z, 0)^2
//   clamped gate : g' = min(gate, limit), u' = clamp(up, -limit, limit); out = g' sigmoid(alpha g') (u' + 1), packed like
//                  the gated SiLU
//   gated GELU   : out = gelu_tanh(gate) * up, packed like the gated SiLU
//   sigmoid gate : y *= sigmoid(z) in place, z a strided view of pre-activation gates
// Reference: none (the reference has no model code).
#include "../common/dtype.cuh"

namespace llmctl {

template <typename T>
__global__ void __launch_bounds__(256)
xielu_kernel(const T* __restrict__ z, T* __restrict__ out, long long n, float a_pos, float a_neg) {
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const float v = to_f32(z[i]);
    const float r = v > 0.f ? a_pos * v * v + 0.5f * v : a_neg * (expm1f(v) - v) + 0.5f * v;
    out[i] = from_f32<T>(r);
  }
}

// x * sigmoid(z).  bf16 operands carry 8 bits, so the hardware's exponential and reciprocal are exact enough there.
template <typename T>
__device__ __forceinline__ float times_sigmoid(float x, float z) {
  if (sizeof(T) == 2) return __fdividef(x, 1.f + __expf(-fmaxf(z, -80.f)));
  return x / (1.f + expf(-z));
}

template <typename T>
struct GateSilu {
  __device__ __forceinline__ float operator()(float g, float u) const { return times_sigmoid<T>(g, g) * u; }
};
// tanh form of GELU: 0.5 g (1 + tanh(y)) = g sigmoid(2 y), y = sqrt(2/pi) (g + 0.044715 g^3)
template <typename T>
struct GateGelu {
  __device__ __forceinline__ float operator()(float g, float u) const {
    return times_sigmoid<T>(g, 1.5957691216057308f * (g + 0.044715f * g * g * g)) * u;
  }
};
template <typename T>
struct GateClamped {
  float limit, alpha;
  __device__ __forceinline__ float operator()(float g, float u) const {
    g = fminf(g, limit);
    return times_sigmoid<T>(g, alpha * g) * (fminf(fmaxf(u, -limit), limit) + 1.f);
  }
};

// out = act(gate, up) on a packed [rows, 2F] activation (gate first, row stride ld).  VEC: numbers per step (8: 16 or 32 bytes).
template <typename T, int VEC, typename Act>
__global__ void __launch_bounds__(256)
gated_kernel(const T* __restrict__ gu, long long ld, T* __restrict__ out, long long groups, int F, Act act) {
  const int per_row = F / VEC;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < groups;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = groups <= 0x7fffffffLL ? static_cast<unsigned>(i) / static_cast<unsigned>(per_row) : i / per_row;
    const int c = static_cast<int>(i - r * per_row) * VEC;
    const T* g = gu + r * ld + c;
    T* o = out + r * F + c;
    if constexpr (VEC == 1) {
      o[0] = from_f32<T>(act(to_f32(g[0]), to_f32(g[F])));
    } else {
      float a[VEC], b[VEC];
      load8_f32(g, a);
      load8_f32(g + F, b);
#pragma unroll
      for (int j = 0; j < VEC; ++j) a[j] = act(a[j], b[j]);
      store8_f32(o, a);
    }
  }
}

// y[r, c] *= sigmoid(z[r, c]) in place; z is a strided view (row stride ldz) of pre-activation gates
template <typename T>
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(T* __restrict__ y, const T* __restrict__ z, long long ldz, int rows, int F) {
  const long long n = static_cast<long long>(rows) * F;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / F;
    const int c = static_cast<int>(i % F);
    y[i] = from_f32<T>(to_f32(y[i]) / (1.f + expf(-to_f32(z[r * ldz + c]))));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) relu_squared_kernel(const T* __restrict__ z, T* __restrict__ out, long long n) {
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const float v = fmaxf(to_f32(z[i]), 0.f);
    out[i] = from_f32<T>(v * v);
  }
}

// in place over a [rows, F] view with row stride ld
template <typename T>
__global__ void __launch_bounds__(256) tanh_kernel(T* __restrict__ z, long long ld, int rows, int F) {
  const long long n = static_cast<long long>(rows) * F;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    T* p = z + i / F * ld + i % F;
    *p = from_f32<T>(tanhf(to_f32(*p)));
  }
}

static inline int grid_for(long long n) {
  long long b = (n + 255) / 256;
  if (b > kNumSMs * 16) b = kNumSMs * 16;
  return static_cast<int>(b);
}

template <typename T, typename Act>
static void launch_gated(const T* gu, long long ld, T* out, int rows, int F, Act act, cudaStream_t s) {
  const bool vec = F % 8 == 0 && ld % 8 == 0 && ((reinterpret_cast<uintptr_t>(gu) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const long long groups = static_cast<long long>(rows) * F / (vec ? 8 : 1);
  if (vec) gated_kernel<T, 8, Act><<<grid_for(groups), 256, 0, s>>>(gu, ld, out, groups, F, act);
  else gated_kernel<T, 1, Act><<<grid_for(groups), 256, 0, s>>>(gu, ld, out, groups, F, act);
}

}  // namespace llmctl

using namespace llmctl;

LLMCTL_API int llmctl_xielu(const void* z, void* out, int is_fp32, long long n, float a_pos, float a_neg, void* stream) {
  LLMCTL_BEGIN();
  if (n == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (xielu_kernel<T><<<grid_for(n), 256, 0, (cudaStream_t)stream>>>((const T*)z, (T*)out, n, a_pos, a_neg)));
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_gated_silu(const void* gate_up, long long ld, void* out, int is_fp32, int rows, int F, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(ld >= 2LL * F);
  if (rows == 0 || F == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (launch_gated<T>((const T*)gate_up, ld, (T*)out, rows, F, GateSilu<T>{}, (cudaStream_t)stream)));
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_gated_gelu_tanh(const void* gate_up, long long ld, void* out, int is_fp32, int rows, int F, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(ld >= 2LL * F);
  if (rows == 0 || F == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (launch_gated<T>((const T*)gate_up, ld, (T*)out, rows, F, GateGelu<T>{}, (cudaStream_t)stream)));
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_sigmoid_gate(void* y, const void* z, long long ldz, int is_fp32, int rows, int F, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(ldz >= F);
  if (rows == 0 || F == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (sigmoid_gate_kernel<T><<<grid_for(static_cast<long long>(rows) * F), 256, 0, (cudaStream_t)stream>>>(
                                        (T*)y, (const T*)z, ldz, rows, F)));
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_gated_clamped(const void* gate_up, long long ld, void* out, int is_fp32, int rows, int F, float limit, float alpha,
                                    void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(ld >= 2LL * F && limit > 0.f);
  if (rows == 0 || F == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (launch_gated<T>((const T*)gate_up, ld, (T*)out, rows, F, GateClamped<T>{limit, alpha}, (cudaStream_t)stream)));
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_relu_squared(const void* z, void* out, int is_fp32, long long n, void* stream) {
  LLMCTL_BEGIN();
  if (n == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (relu_squared_kernel<T><<<grid_for(n), 256, 0, (cudaStream_t)stream>>>((const T*)z, (T*)out, n)));
  LLMCTL_RETURN_LAST();
}

// z <- tanh(z) in place, [rows, F] with row stride ld
LLMCTL_API int llmctl_tanh(void* z, long long ld, int is_fp32, int rows, int F, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(ld >= F);
  if (rows == 0 || F == 0) return 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (tanh_kernel<T><<<grid_for(static_cast<long long>(rows) * F), 256, 0, (cudaStream_t)stream>>>((T*)z, ld, rows, F)));
  LLMCTL_RETURN_LAST();
}
