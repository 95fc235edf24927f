// Serial scan and single-token step of recurrences with a matrix state S [d, e] per head, fp32, shared by matrix_state.cu (gated
// delta rules, kinds 0 and 1; outer products with a bonus, kind 2) and retention.cu (kind 3):
//
//   kind 0, 1:  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q        g per head (0) or per head and key row (1)
//   kind 2:     o = S^T q + bonus v;  S <- diag(g) S + k v^T
//   kind 3:     S <- g S + k v^T;  o = S^T q                                         g per head
//
// The scan reads what a prepare pass left in MsWork; the step forms its token's vectors itself.
#pragma once
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

// kinds 1 and 2 have a decay per key row, the others one per head; the delta rules subtract what the state already holds
static inline __host__ __device__ constexpr bool ms_row_decay(int kind) { return kind == 1 || kind == 2; }
static inline __host__ __device__ constexpr bool ms_is_delta(int kind) { return kind <= 1; }

// A token's prepared numbers as a lane holds them.
template <int NP, int CPL, int KIND>
struct ScanToken {
  f32x2 k[NP], q[NP], d[ms_row_decay(KIND) ? NP : 1];
  float4 sc;
  float v[CPL];
};

// KIND 0: delta rule, decay per head; 1: delta rule, decay per key row; 2: outer products with a bonus; 3: retention.
// A lane owns columns c0 .. c0 + CPL - 1 and the rows (i LPC + sub) 4 .. + 3, i < RPT / 4; the CTA 16 CPL columns.
template <int RPT, int LPC, int CPL, int KIND>
__global__ void __launch_bounds__(LPC * 16)
matrix_scan_kernel(const MatrixScanParams p) {
  constexpr int TC = kMsTC, DP = RPT * LPC, NG = 32 / LPC, NT = LPC * 16, NP = RPT / 2, COLS = 16 * CPL;
  constexpr int NROW = ms_row_decay(KIND) ? 3 : 2, STAGE = TC * (DP * NROW + COLS + 4);
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
      if (ms_row_decay(KIND)) cp_async_16(sd + tok * DP + c, p.w.dm + ((tb + tok) * H + h) * DP + c);
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
        if (ms_row_decay(KIND)) ld_pairs(sd + tok * DP + i * 2 * LPC, w.d[ms_row_decay(KIND) ? i : 0], w.d[ms_row_decay(KIND) ? i + 1 : 0]);
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
          S[c][i] = fma2(ms_row_decay(KIND) ? w.d[ms_row_decay(KIND) ? i : 0] : dh, S[c][i], S[c][i]);
          if (KIND == 3) qa[c][i & 1] = fma2(w.q[i], S[c][i], qa[c][i & 1]);
          if (ms_is_delta(KIND)) ka[c][i & 1] = fma2(w.k[i], S[c][i], ka[c][i & 1]);
        }
      float u[CPL], o[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        u[c] = w.v[c];
        if (ms_is_delta(KIND)) {
          const float2 x = upk(ka[c][0]), y = upk(ka[c][1]);
          o[c] = (x.x + y.x) + (x.y + y.y);
        }
      }
      if (ms_is_delta(KIND)) {               // the read-out's products fill the waits of these shuffles
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
  const void* r;              // kinds 2, 3: r (queries), k, v (row strides ldr, ldk, ldv)
  const void* k;
  const void* v;
  long long ldx, ldr, ldk, ldv;
  const float* conv_w;        // kinds 0, 1
  float* conv_state;
  int taps;
  const void* z;
  long long ldz;
  const float* z_bias;        // dt_bias, or w0 of kind 2
  const float* speed;         // [H], kinds 0, 1; kind 3: decay minus one
  const float* bonus;         // [H d], kind 2
  const void* b;              // [T, H], kinds 0, 1
  long long ldb;
  const int* portions;
  float* state;               // [slots, H, d, e]
  const float* norm_w;        // [e] (norm_stride 0) or [H, e] (norm_stride e), null: no weight
  int norm_stride;
  const void* gate;           // [T, H e] pre-activation
  long long ldg;
  int gate_kind;              // 0: silu, 1: sigmoid
  float eps;
  void* out;                  // [T, H e]
  int H, G, d, e;
  const int* positions;       // kind 3: [T], frequencies [rot / 2]
  const float* freq;
  int rot;
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
  float* cst = (ms_is_delta(KIND) && slot >= 0) ? p.conv_state + static_cast<long long>(slot) * (p.taps - 1) * C : nullptr;

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
      } else if (KIND == 3) {
        const T* qr = static_cast<const T*>(p.r) + t * p.ldr + g * d;
        const T* kr = static_cast<const T*>(p.k) + t * p.ldk + g * d;
        q = to_f32(qr[tid]), k = to_f32(kr[tid]);
        if (tid < p.rot) {
          const int half = p.rot >> 1;
          const bool second = tid >= half;
          const int o = second ? tid - half : tid + half;
          float s, c;
          sincosf(static_cast<float>(p.positions[t]) * p.freq[second ? o : tid], &s, &c);
          if (!second) s = -s;
          q = q * c + to_f32(qr[o]) * s;
          k = k * c + to_f32(kr[o]) * s;
        }
        k *= 1.f / sqrtf(static_cast<float>(d));
      } else {
        const T* x = static_cast<const T*>(p.x) + t * p.ldx;
        q = ms_conv_step(x, p.conv_w, cst, has, p.taps, C, g * d + tid);
        k = ms_conv_step(x, p.conv_w, cst, has, p.taps, C, (G + g) * d + tid);
      }
    }
    if (KIND == 2) {
      qk = block_sum(tid < d ? q * k * p.bonus[g * d + tid] : 0.f, red);
    } else if (KIND == 3) {
      qk = block_sum(q * k, red);
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
    if (KIND == 3) dm = p.speed[h];
    if (ms_is_delta(KIND)) {
      beta = ms_sigmoid(to_f32(static_cast<const T*>(p.b)[t * p.ldb + h]));
      if (KIND == 0) dm = expm1f(-p.speed[h] * ms_softplus(to_f32(static_cast<const T*>(p.z)[t * p.ldz + h]) + p.z_bias[h]));
    }
    if (ms_row_decay(KIND) && tid < DP) {
      float v = 0.f;
      if (tid < d) {
        const float z = to_f32(static_cast<const T*>(p.z)[t * p.ldz + h * d + tid]) + p.z_bias[h * d + tid];
        v = KIND == 2 ? expm1f(-expf(z)) : expm1f(-p.speed[h] * ms_softplus(z));
      }
      sd[tid] = v;
    }
    for (int c = tid; c < e; c += 256) {
      if (!ms_is_delta(KIND)) sv[c] = to_f32(static_cast<const T*>(p.v)[t * p.ldv + h * e + c]);
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
        const float kk = sk[row], qq = sq[row], dd = ms_row_decay(KIND) ? sd[row] : dm;
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          if (KIND == 2) qa[j] += qq * S[i][j];
          S[i][j] = fmaf(dd, S[i][j], S[i][j]);
          if (ms_is_delta(KIND)) ka[j] += kk * S[i][j];
          if (KIND != 2) qa[j] += qq * S[i][j];
        }
      }
      if (ms_is_delta(KIND)) ms_stv<VEC>(part + (warp * 2) * TILE + lane * VEC, ka);
      ms_stv<VEC>(part + (warp * 2 + 1) * TILE + lane * VEC, qa);
      __syncthreads();
      float u[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) u[j] = col + j < e ? sv[col + j] : 0.f;
      if (ms_is_delta(KIND)) {
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
      static_cast<T*>(p.out)[(t * H + h) * e + c] = from_f32<T>(so[c] * f * (p.norm_w ? p.norm_w[h * p.norm_stride + c] : 1.f) * act);
    }
  }
}

template <int RPT, int LPC, int CPL, int KIND>
static int launch_matrix_scan_cols(const MatrixScanParams& p, int nportions, cudaStream_t s) {
  constexpr int DP = RPT * LPC, COLS = 16 * CPL;
  const size_t smem = sizeof(float) * (2 * kMsTC * (static_cast<size_t>(DP) * (ms_row_decay(KIND) ? 3 : 2) + COLS + 4) + 2 * kMsTC * COLS);
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
