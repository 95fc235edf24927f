// Mixture-of-experts feed-forward: routing, token permutation, grouped expert GEMMs and the weighted combine, with no
// host synchronisation anywhere (expert loads stay on the device).  bf16 or fp32 activations / weights; router
// arithmetic, accumulators and the combine are fp32.
//
//   llmctl_moe_route   : per token, logits = Wr x (fp32), score = sigmoid or softmax over experts, the `top` largest
//                        (ties: lowest index), optionally renormalised to sum 1; optional per-token gate
//                        sigmoid(wg . x) of a shared expert; counts tokens per expert.  Optionally the CHOICE is made on
//                        score + correction[e] (the weights stay the plain scores) and restricted to the
//                        `keep_groups` of `n_groups` equal groups of neighbouring experts whose group score is largest
//                        (the others count as minus infinity); a group's score is its best choice score or the sum of
//                        its two best.  The weights may be multiplied by a constant.  Expert ids >= the number of experts with
//                        weights (`E` of plan / permute) are identity experts: they get no rows in the permuted
//                        buffer and the combine adds weight * (the token's input) for them.
//   llmctl_moe_plan    : one CTA: per-expert row offsets in the permuted buffer, every expert's segment padded to a
//                        multiple of the GEMM's row tile, and the tile -> expert map.
//   llmctl_moe_permute : copies every (token, choice) pair's input row into its expert's segment, multiplied by the
//                        routing weight when the weight applies to the expert's INPUT (scale_input), and records
//                        where it went.
//   llmctl_grouped_gemm: out[row, :] = A[row, :] W[expert(row)]^T over the permuted rows; a CTA computes a 64 x 64 tile
//                        of one expert (row tiles never straddle experts thanks to the padding).  bf16 with K and N
//                        multiples of 8 runs 64 x 128 tiles on the tensor cores (mma.sync m16n8k16, fp32 accumulation,
//                        next k-slice prefetched into registers); fp32 and odd sizes run the FMA kernel.
//                        bf16 on 128-row tiles can instead run on the tcgen05 GEMM's grouped mode (llmctl_gemm_bf16_grouped,
//                        csrc/gemm/gemm_tcgen05.cu), which reads the same plan.
//   llmctl_moe_combine : y[t] = sum_k (w_k if the weight applies to the OUTPUT) * expert_out[row(t, k)]
//                               + gate[t] * shared_out[t], in a fixed order (deterministic), fp32.
// Reference: none (the reference has no model code).
#include "../common/dtype.cuh"
#include "../common/mma_sync.cuh"

namespace llmctl {

constexpr int kTileM = 64, kTileN = 64, kTileK = 16;

struct RouteParams {
  const float* x;             // [tokens, W] (the residual stream)
  const void* wr;             // [E, W]
  const void* wg;             // [W] or null
  int tokens, W, E, top, softmax_scores, renormalise;
  const float* correction;
  int n_groups, keep_groups, group_best;
  float weight_scale;
  int* ids;
  float* weights;
  float* gate;
  int* counts;
};

constexpr int kRouteExperts = 2;      // router rows a warp reads at a time

// largest (value, lowest index) of the warp; index -1: none
__device__ __forceinline__ void warp_best(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (oi >= 0 && (i < 0 || ov > v || (ov == v && oi < i))) v = ov, i = oi;
  }
}

// One warp: scores of a token (score[0 .. E)) -> ids and weights.
__device__ __forceinline__ void route_choose(const RouteParams& p, float* score, float* choice, long long tok, int lane) {
  const int E = p.E, top = p.top;
  if (p.softmax_scores == 2) {
    // raw logits decide the choice; the weights are a softmax over the chosen logits only (below)
  } else if (p.softmax_scores) {
    float m = -INFINITY, z = 0.f;
    for (int e = lane; e < E; e += 32) m = fmaxf(m, score[e]);
    m = warp_max(m);
    for (int e = lane; e < E; e += 32) z += (score[e] = expf(score[e] - m));
    z = warp_sum(z);
    for (int e = lane; e < E; e += 32) score[e] /= z;
  } else {
    for (int e = lane; e < E; e += 32) score[e] = 1.f / (1.f + expf(-score[e]));
  }
  for (int e = lane; e < E; e += 32) choice[e] = score[e] + (p.correction ? p.correction[e] : 0.f);
  __syncwarp();
  if (p.n_groups > 1 && p.keep_groups < p.n_groups) {
    // a group's score is its largest choice score, or the sum of its two largest; groups outside the best `keep_groups` cannot be chosen
    const int gs = E / p.n_groups;
    float gv[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {                      // n_groups <= 64
      const int gi = lane + 32 * j;
      gv[j] = -INFINITY;
      float second = -INFINITY;
      if (gi < p.n_groups) {
        for (int e = gi * gs; e < (gi + 1) * gs; ++e) {
          second = fmaxf(second, fminf(gv[j], choice[e]));
          gv[j] = fmaxf(gv[j], choice[e]);
        }
        if (p.group_best == 2 && gs > 1) gv[j] += second;
      }
    }
    unsigned long long kept = 0ull;
    for (int r = 0; r < p.keep_groups; ++r) {
      float v = -INFINITY;
      int i = -1;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int gi = lane + 32 * j;
        if (gi < p.n_groups && !(kept >> gi & 1ull) && (i < 0 || gv[j] > v)) v = gv[j], i = gi;
      }
      warp_best(v, i);
      kept |= 1ull << i;
    }
    for (int e = lane; e < E; e += 32)
      if (!(kept >> (e / gs) & 1ull)) choice[e] = -INFINITY;
    __syncwarp();
  }
  float total = 0.f, first = 0.f;
  for (int k = 0; k < top; ++k) {
    float v = -INFINITY;
    int best = -1;
    for (int e = lane; e < E; e += 32)
      if (choice[e] > v) v = choice[e], best = e;
    warp_best(v, best);
    if (best < 0) {                                    // fewer choosable experts than `top` (NaN scores): first unchosen one
      for (int e = 0; e < E && best < 0; ++e) {
        bool taken = false;
        for (int kk = 0; kk < k; ++kk) taken |= p.ids[tok * top + kk] == e;
        if (!taken) best = e;
      }
    }
    const float w = score[best];
    if (k == 0) first = w;
    total += p.softmax_scores == 2 ? expf(w - first) : w;      // the first choice is the largest logit
    if (lane == 0) {
      p.ids[tok * top + k] = best;
      p.weights[tok * top + k] = w;
      choice[best] = -INFINITY;
      atomicAdd(&p.counts[best], 1);
    }
    __syncwarp();
  }
  if (p.softmax_scores != 2 && !p.renormalise && p.weight_scale == 1.f) return;
  for (int k = lane; k < top; k += 32) {
    float w = p.weights[tok * top + k];
    if (p.softmax_scores == 2) w = expf(w - first) / total;
    else if (p.renormalise) w /= total + 1e-20f;
    p.weights[tok * top + k] = w * p.weight_scale;
  }
}

constexpr int kRouteTokens = 8, kRouteCols = 256, kRouteStages = 4;

// Logits of eight tokens against two router rows per warp at a time: the tokens' columns stream through shared memory (cp.async,
// four stages of 256 columns), the next router numbers are asked for before the current ones are used.  A lane adds up the same
// products in the same order as in moe_route_kernel<T, 1, 4>.
template <typename T>
__device__ __forceinline__ void route_logits_staged(const RouteParams& p, float* xs, float* score, long long tok0, int nt) {
  constexpr int TT = kRouteTokens, CH = kRouteCols, NS = kRouteStages, NC = CH / 128;
  const int W = p.W, E = p.E, rows = E + (p.wg ? 1 : 0), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarp = blockDim.x >> 5;
  const int nst = (W + CH - 1) / CH;
  auto stage = [&](int i) {
    float* dst = xs + (i % NS) * TT * CH;
    for (int k = tid; k < TT * CH / 4; k += blockDim.x) {
      const int t = k / (CH / 4), c = i * CH + k % (CH / 4) * 4;
      if (c < W) cp_async_16(dst + t * CH + k % (CH / 4) * 4, p.x + (tok0 + min(t, nt - 1)) * W + c);
    }
  };
  for (int e0 = warp * kRouteExperts; e0 - warp * kRouteExperts < rows; e0 += nwarp * kRouteExperts) {      // every warp takes part in the staging
    const bool on = e0 < rows;
    const T* w[kRouteExperts];
#pragma unroll
    for (int j = 0; j < kRouteExperts; ++j) {
      const int e = min(e0 + j, rows - 1);
      w[j] = (e < E ? static_cast<const T*>(p.wr) + static_cast<long long>(e) * W : static_cast<const T*>(p.wg)) + lane * 4;
    }
    float acc[TT][kRouteExperts];
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
      for (int j = 0; j < kRouteExperts; ++j) acc[t][j] = 0.f;
    __syncthreads();                                   // the previous round's readers are done
    for (int i = 0; i < NS - 1; ++i) {
      if (i < nst) stage(i);
      cp_async_commit();
    }
    float wn[kRouteExperts][4];
#pragma unroll
    for (int j = 0; j < kRouteExperts; ++j)
      if (on && lane * 4 < W) load_vec<4>(w[j], wn[j]);
    for (int i = 0; i < nst; ++i) {
      asm volatile("cp.async.wait_group %0;\n" ::"n"(kRouteStages - 2) : "memory");
      __syncthreads();                                 // stage i has landed; everyone is done with stage i - 1
      if (i + NS - 1 < nst) stage(i + NS - 1);
      cp_async_commit();
      const float* x = xs + (i % NS) * TT * CH + lane * 4;
#pragma unroll
      for (int ch = 0; ch < NC; ++ch) {
        const int c = i * CH + ch * 128 + lane * 4;
        if (!on || c >= W) continue;
        float wv[kRouteExperts][4];
#pragma unroll
        for (int j = 0; j < kRouteExperts; ++j) {
#pragma unroll
          for (int k = 0; k < 4; ++k) wv[j][k] = wn[j][k];
          if (c + 128 < W) load_vec<4>(w[j] + i * CH + ch * 128 + 128, wn[j]);
        }
#pragma unroll
        for (int t = 0; t < TT; ++t) {
          float xv[4];
          load_vec<4>(x + t * CH + ch * 128, xv);
#pragma unroll
          for (int j = 0; j < kRouteExperts; ++j)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[t][j] = fmaf(xv[k], wv[j][k], acc[t][j]);
        }
      }
    }
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
      for (int j = 0; j < kRouteExperts; ++j) {
        const float s = warp_sum(acc[t][j]);
        if (lane == 0 && t < nt && e0 + j < rows) {
          if (e0 + j < E) score[t * E + e0 + j] = s;
          else p.gate[tok0 + t] = 1.f / (1.f + expf(-s));
        }
      }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
moe_route_staged_kernel(const RouteParams p) {
  extern __shared__ __align__(16) float route_smem[];  // stages, [TT][E] scores, [TT][E] choice scores
  constexpr int TT = kRouteTokens;
  const long long tok0 = static_cast<long long>(blockIdx.x) * TT;
  const int nt = static_cast<int>(min(static_cast<long long>(TT), p.tokens - tok0));
  float* score = route_smem + kRouteStages * TT * kRouteCols;
  route_logits_staged<T>(p, route_smem, score, tok0, nt);
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
  for (int t = warp; t < nt; t += nwarp) route_choose(p, score + t * p.E, score + (TT + t) * p.E, tok0 + t, lane);
}

// A CTA routes TT tokens: a warp holds two router rows against all of them at a time (the order of a logit's sum depends on W and
// VEC alone), then every warp chooses for one token.
template <typename T, int TT, int VEC>
__global__ void __launch_bounds__(256)
moe_route_kernel(const RouteParams p) {
  extern __shared__ float route_smem[];                // [TT][E] scores, [TT][E] choice scores
  const int W = p.W, E = p.E, rows = E + (p.wg ? 1 : 0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
  const long long tok0 = static_cast<long long>(blockIdx.x) * TT;
  const int nt = static_cast<int>(min(static_cast<long long>(TT), p.tokens - tok0));
  for (int e0 = warp * kRouteExperts; e0 < rows; e0 += nwarp * kRouteExperts) {
    const T* w[kRouteExperts];
#pragma unroll
    for (int j = 0; j < kRouteExperts; ++j) {
      const int e = min(e0 + j, rows - 1);
      w[j] = e < E ? static_cast<const T*>(p.wr) + static_cast<long long>(e) * W : static_cast<const T*>(p.wg);
    }
    float acc[TT][kRouteExperts];
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
      for (int j = 0; j < kRouteExperts; ++j) acc[t][j] = 0.f;
#pragma unroll(TT == 1 ? 4 : 1)
    for (int c = lane * VEC; c < W; c += 32 * VEC) {
      float wv[kRouteExperts][VEC];
#pragma unroll
      for (int j = 0; j < kRouteExperts; ++j) load_vec<VEC>(w[j] + c, wv[j]);
#pragma unroll
      for (int t = 0; t < TT; ++t) {
        float xv[VEC];
        load_vec<VEC>(p.x + (tok0 + min(t, nt - 1)) * W + c, xv);
#pragma unroll
        for (int j = 0; j < kRouteExperts; ++j)
#pragma unroll
          for (int i = 0; i < VEC; ++i) acc[t][j] = fmaf(xv[i], wv[j][i], acc[t][j]);
      }
    }
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
      for (int j = 0; j < kRouteExperts; ++j) {
        const float s = warp_sum(acc[t][j]);
        if (lane == 0 && t < nt && e0 + j < rows) {
          if (e0 + j < E) route_smem[t * E + e0 + j] = s;
          else p.gate[tok0 + t] = 1.f / (1.f + expf(-s));
        }
      }
  }
  __syncthreads();
  for (int t = warp; t < nt; t += nwarp) route_choose(p, route_smem + t * E, route_smem + (TT + t) * E, tok0 + t, lane);
}

template <typename T, int TT>
static int launch_route(const RouteParams& p, bool vec, cudaStream_t s) {
  const size_t smem = 2 * static_cast<size_t>(TT) * p.E * sizeof(float);
  auto kern = vec ? moe_route_kernel<T, TT, 4> : moe_route_kernel<T, TT, 1>;
  if (smem > 46 * 1024) LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kern<<<(p.tokens + TT - 1) / TT, 256, smem, s>>>(p);
  return 0;
}

// meta: int32 [2 * E + 2 + max_tiles] = { offsets[E] | cursor[E] | num_tiles | padded rows | tile_expert[max_tiles] }
__global__ void moe_plan_kernel(const int* __restrict__ counts, int E, int* __restrict__ meta, int max_tiles, int tile_m) {
  if (threadIdx.x != 0) return;
  int* offsets = meta;
  int* cursor = meta + E;
  int* tile_expert = meta + 2 * E + 2;
  int row = 0, tile = 0;
  for (int e = 0; e < E; ++e) {
    offsets[e] = row;
    cursor[e] = 0;
    const int nt = (counts[e] + tile_m - 1) / tile_m;
    for (int i = 0; i < nt && tile < max_tiles; ++i) tile_expert[tile++] = e;
    row += nt * tile_m;
  }
  meta[2 * E] = tile;
  meta[2 * E + 1] = row;
}

// One CTA per token, all its choices.  dst rows of a segment beyond the expert's count are never read back.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
moe_permute_kernel(const float* __restrict__ x, int W, const int* __restrict__ ids, const float* __restrict__ weights,
                   int scale_input, int* __restrict__ meta, int E, int top, int* __restrict__ pair_row, T* __restrict__ xs) {
  extern __shared__ int s_row[];                       // [top] rows, then [top] weights
  float* s_w = reinterpret_cast<float*>(s_row + top);
  const long long tok = blockIdx.x;
  for (int k = threadIdx.x; k < top; k += blockDim.x) {
    const int e = ids[tok * top + k];
    const int row = e < E ? meta[e] + atomicAdd(&meta[E + e], 1) : -1;       // ids >= E: identity experts, no row
    s_row[k] = pair_row[tok * top + k] = row;
    s_w[k] = scale_input ? weights[tok * top + k] : 1.f;
  }
  __syncthreads();
  const float* src = x + tok * W;
  for (int c = threadIdx.x * VEC; c < W; c += blockDim.x * VEC) {
    float v[VEC];
    load_vec<VEC>(src + c, v);
    for (int k = 0; k < top; ++k) {
      if (s_row[k] < 0) continue;
      float o[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = s_w[k] * v[i];
      store_vec<VEC>(xs + static_cast<long long>(s_row[k]) * W + c, o);
    }
  }
}

// A: [padded rows, K] (row stride lda); Wt: [E, N, K] contiguous; out: [padded rows, N].
// 256 threads, each a 4 x 4 block of the 64 x 64 tile; fp32 accumulation whatever T.
template <typename T>
__global__ void __launch_bounds__(256)
grouped_gemm_kernel(const T* __restrict__ A, long long lda, const T* __restrict__ Wt, T* __restrict__ out, long long ldo,
                    int N, int K, const int* __restrict__ meta, int E) {
  const int tile = blockIdx.x;
  if (tile >= meta[2 * E]) return;
  const int e = meta[2 * E + 2 + tile];
  const long long row0 = static_cast<long long>(tile) * kTileM;
  const int n0 = blockIdx.y * kTileN;
  const T* Bw = Wt + static_cast<long long>(e) * N * K;
  __shared__ float As[kTileK][kTileM + 4];
  __shared__ float Bs[kTileK][kTileN + 4];
  const int tid = threadIdx.x;
  const int tr = (tid / 16) * 4, tc = (tid % 16) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kTileK) {
    for (int idx = tid; idx < kTileM * kTileK; idx += 256) {
      const int r = idx / kTileK, k = idx % kTileK;
      As[k][r] = (k0 + k < K) ? to_f32(A[(row0 + r) * lda + k0 + k]) : 0.f;
      const int n = n0 + r;
      Bs[k][r] = (k0 + k < K && n < N) ? to_f32(Bw[static_cast<long long>(n) * K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTileK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = As[k][tr + i];
        b[i] = Bs[k][tc + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n0 + tc + j < N) out[(row0 + tr + i) * ldo + n0 + tc + j] = from_f32<T>(acc[i][j]);
}

// bf16 tensor-core variant: 64 x 128 tile, 8 warps as 2 (rows) x 4 (columns), each 32 x 32.
constexpr int kTcN = 128, kTcK = 32, kTcLd = kTcK + 8;

__global__ void __launch_bounds__(256)
grouped_gemm_tc_kernel(const __nv_bfloat16* __restrict__ A, long long lda, const __nv_bfloat16* __restrict__ Wt,
                       __nv_bfloat16* __restrict__ out, long long ldo, int N, int K, const int* __restrict__ meta, int E) {
  const int tile = blockIdx.x;
  if (tile >= meta[2 * E]) return;
  const int e = meta[2 * E + 2 + tile];
  const long long row0 = static_cast<long long>(tile) * kTileM;
  const int n0 = blockIdx.y * kTcN;
  const __nv_bfloat16* Bw = Wt + static_cast<long long>(e) * N * K;
  __shared__ __align__(16) __nv_bfloat16 As[kTileM * kTcLd];
  __shared__ __align__(16) __nv_bfloat16 Bs[kTcN * kTcLd];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int wm = warp >> 2, wn = warp & 3;
  const int lr = tid >> 2, lv = tid & 3;          // this thread's row and 8-element slice within a k-slice
  float acc[2][4][4] = {};
  uint4 ra, rb[2];
  auto fetch = [&](int k0) {
    const int k = k0 + lv * 8;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    ra = k < K ? *reinterpret_cast<const uint4*>(A + (row0 + lr) * lda + k) : zero;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int n = n0 + lr + 64 * i;
      rb[i] = (k < K && n < N) ? *reinterpret_cast<const uint4*>(Bw + static_cast<long long>(n) * K + k) : zero;
    }
  };
  fetch(0);
  for (int k0 = 0; k0 < K; k0 += kTcK) {
    *reinterpret_cast<uint4*>(As + lr * kTcLd + lv * 8) = ra;
    *reinterpret_cast<uint4*>(Bs + lr * kTcLd + lv * 8) = rb[0];
    *reinterpret_cast<uint4*>(Bs + (lr + 64) * kTcLd + lv * 8) = rb[1];
    __syncthreads();
    if (k0 + kTcK < K) fetch(k0 + kTcK);
#pragma unroll
    for (int kk = 0; kk < kTcK; kk += 16) {
      uint32_t a[2][4];
#pragma unroll
      for (int mi = 0; mi < 2; ++mi) load_a_frag(a[mi], As, kTcLd, 32 * wm + 16 * mi, kk, lane);
#pragma unroll
      for (int ni = 0; ni < 4; ++ni) {
        uint32_t b[2];
        load_b_frag_nk(b, Bs, kTcLd, 32 * wn + 8 * ni, kk, lane);
#pragma unroll
        for (int mi = 0; mi < 2; ++mi) mma_bf16_16816(acc[mi][ni], a[mi], b);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int mi = 0; mi < 2; ++mi)
#pragma unroll
    for (int ni = 0; ni < 4; ++ni) {
      const int col = n0 + 32 * wn + 8 * ni + 2 * t;
      if (col < N) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const long long row = row0 + 32 * wm + 16 * mi + g + 8 * half;
          *reinterpret_cast<__nv_bfloat162*>(out + row * ldo + col) =
              __floats2bfloat162_rn(acc[mi][ni][2 * half], acc[mi][ni][2 * half + 1]);
        }
      }
    }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
moe_combine_kernel(const T* __restrict__ expert_out, int W, const int* __restrict__ pair_row,
                   const float* __restrict__ weights, int top, int scale_output, const T* __restrict__ shared_out,
                   const float* __restrict__ gate, const float* __restrict__ identity_in, float* __restrict__ y) {
  extern __shared__ int s_row[];                       // [top] rows, then [top] weights
  float* s_w = reinterpret_cast<float*>(s_row + top);
  const long long tok = blockIdx.x;
  for (int k = threadIdx.x; k < top; k += blockDim.x) {
    s_row[k] = pair_row[tok * top + k];
    s_w[k] = weights[tok * top + k];
  }
  __syncthreads();
  const float g = gate ? gate[tok] : 1.f;
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; c < W; c += gridDim.y * blockDim.x * VEC) {
    float a[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) a[i] = 0.f;
#pragma unroll 4
    for (int k = 0; k < top; ++k) {
      const int row = s_row[k];
      float v[VEC];
      if (row < 0) load_vec<VEC>(identity_in + tok * W + c, v);       // an identity expert: weight times the token's input
      else load_vec<VEC>(expert_out + static_cast<long long>(row) * W + c, v);
      const float w = (scale_output || row < 0) ? s_w[k] : 1.f;
#pragma unroll
      for (int i = 0; i < VEC; ++i) a[i] += w * v[i];
    }
    if (shared_out) {
      float v[VEC];
      load_vec<VEC>(shared_out + tok * W + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) a[i] += g * v[i];
    }
    store_vec<VEC>(y + tok * W + c, a);
  }
}

}  // namespace llmctl

using namespace llmctl;

LLMCTL_API int llmctl_moe_tile_rows() { return kTileM; }

LLMCTL_API int llmctl_moe_route(const float* x, const void* wr, const void* wg, int is_fp32, int tokens, int W, int E, int top,
                                int softmax_scores, int renormalise, const float* correction, int n_groups, int keep_groups,
                                int group_best, float weight_scale, int* ids, float* weights, float* gate, int* counts, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(E >= 1 && top >= 1 && top <= E && E <= 4096 && (wg == nullptr || gate != nullptr));
  LLMCTL_REQUIRE(n_groups <= 1 || (n_groups <= 64 && E % n_groups == 0 && keep_groups >= 1 && keep_groups <= n_groups &&
                                   keep_groups * (E / n_groups) >= top && (group_best == 1 || group_best == 2)));
  cudaStream_t s = (cudaStream_t)stream;
  LLMCTL_CHECK(cudaMemsetAsync(counts, 0, sizeof(int) * E, s));
  if (tokens == 0) return 0;
  const RouteParams p{x, wr, wg, tokens, W, E, top, softmax_scores, renormalise, correction, n_groups, keep_groups, group_best, weight_scale, ids,
                      weights, gate, counts};
  const uintptr_t al = is_fp32 ? 15 : 7;
  const bool vec = W % 4 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 && ((reinterpret_cast<uintptr_t>(wr) | reinterpret_cast<uintptr_t>(wg)) & al) == 0;
  const bool many = tokens >= 4 * kNumSMs && E <= 1024;          // few tokens: one per CTA, latency counts
  int rc = 0;
  if (many && vec) {
    const size_t smem = (kRouteStages * kRouteTokens * kRouteCols + 2 * static_cast<size_t>(kRouteTokens) * E) * sizeof(float);
    LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
      auto kern = moe_route_staged_kernel<T>;
      if (smem > 46 * 1024) LLMCTL_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
      kern<<<(tokens + kRouteTokens - 1) / kRouteTokens, 256, smem, s>>>(p);
    });
    LLMCTL_RETURN_LAST();
  }
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (rc = many ? launch_route<T, 8>(p, false, s) : launch_route<T, 1>(p, vec, s)));
  if (rc) return rc;
  LLMCTL_RETURN_LAST();
}

// tile_rows: the row tile of the grouped GEMM that will read the plan: llmctl_moe_tile_rows() for llmctl_grouped_gemm,
// 128 for llmctl_gemm_bf16_grouped (which takes tile_expert = meta + 2 E + 2 and num_tiles = meta + 2 E).
LLMCTL_API int llmctl_moe_plan(const int* counts, int E, int* meta, int max_tiles, int tile_rows, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(tile_rows == kTileM || tile_rows == 128);
  moe_plan_kernel<<<1, 32, 0, (cudaStream_t)stream>>>(counts, E, meta, max_tiles, tile_rows);
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_moe_permute(const float* x, int W, const int* ids, const float* weights, int scale_input, int* meta,
                                  int E, int* pair_row, void* xs, int is_fp32, int tokens, int top, void* stream) {
  LLMCTL_BEGIN();
  if (tokens == 0) return 0;
  const bool vec = W % 4 == 0 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (reinterpret_cast<uintptr_t>(xs) & (is_fp32 ? 15 : 7)) == 0;
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    auto kern = vec ? moe_permute_kernel<T, 4> : moe_permute_kernel<T, 1>;
    kern<<<tokens, 256, 2 * top * sizeof(int), (cudaStream_t)stream>>>(x, W, ids, weights, scale_input, meta, E, top, pair_row, (T*)xs);
  });
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_grouped_gemm(const void* A, long long lda, const void* Wt, void* out, long long ldo, int N, int K,
                                   const int* meta, int E, int max_tiles, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  LLMCTL_REQUIRE(N > 0 && K > 0 && lda >= K && ldo >= N);
  if (max_tiles == 0) return 0;
  if (!is_fp32 && K % 8 == 0 && N % 8 == 0 && lda % 8 == 0 && ldo % 2 == 0 && (reinterpret_cast<uintptr_t>(A) & 15) == 0 &&
      (reinterpret_cast<uintptr_t>(Wt) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 3) == 0) {
    grouped_gemm_tc_kernel<<<dim3(max_tiles, (N + kTcN - 1) / kTcN), 256, 0, (cudaStream_t)stream>>>(
        (const __nv_bfloat16*)A, lda, (const __nv_bfloat16*)Wt, (__nv_bfloat16*)out, ldo, N, K, meta, E);
    LLMCTL_RETURN_LAST();
  }
  dim3 grid(max_tiles, (N + kTileN - 1) / kTileN);
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, (grouped_gemm_kernel<T><<<grid, 256, 0, (cudaStream_t)stream>>>(
                                        (const T*)A, lda, (const T*)Wt, (T*)out, ldo, N, K, meta, E)));
  LLMCTL_RETURN_LAST();
}

LLMCTL_API int llmctl_moe_combine(const void* expert_out, int W, const int* pair_row, const float* weights, int top,
                                  int scale_output, const void* shared_out, const float* gate, const float* identity_in,
                                  float* y, int tokens, int is_fp32, void* stream) {
  LLMCTL_BEGIN();
  if (tokens == 0) return 0;
  const uintptr_t al = is_fp32 ? 15 : 7;
  const bool vec = W % 4 == 0 && ((reinterpret_cast<uintptr_t>(expert_out) | reinterpret_cast<uintptr_t>(shared_out)) & al) == 0 &&
                   ((reinterpret_cast<uintptr_t>(identity_in) | reinterpret_cast<uintptr_t>(y)) & 15) == 0;
  const dim3 grid(tokens, tokens < kNumSMs ? (W / (vec ? 4 : 1) + 255) / 256 : 1);      // few tokens: a row's columns over several CTAs
  LLMCTL_DISPATCH_DTYPE(is_fp32, T, {
    auto kern = vec ? moe_combine_kernel<T, 4> : moe_combine_kernel<T, 1>;
    kern<<<grid, 256, 2 * top * sizeof(int), (cudaStream_t)stream>>>((const T*)expert_out, W, pair_row, weights, top, scale_output, (const T*)shared_out,
                                                                     gate, identity_in, y);
  });
  LLMCTL_RETURN_LAST();
}
