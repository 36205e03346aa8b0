// Linear attention with a constant decay per head (lightning attention), for sm_100a:
//     S_t = decay S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t,   q, k, v = silu of the packed projection (or as given)
//
//   decayed_step        one token per row: the fp32 state is read and written once
//   decayed_chunks      a call's tokens in chunks of 64 on the tensor cores (bf16, head widths up to 128 in multiples of 8)
//   decayed_sequence    a call's tokens one after another, any head widths, fp32 arithmetic (the exact form; it also serves fp32 models)
//
// The packed projection is [rows, S, H dk | H dk | H dv] (q, k, v; heads inside each).  `state` [store rows, H, dk, dv] fp32 stays on the
// device between calls; a call row whose first position is 0 starts from zero, positions below 0 are padding (they come last in a row,
// change no state and give zero outputs).  Compiled without fast math.
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/mma_bf16.cuh"

namespace dewb {
namespace decayed {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float silu(float x, float*) { return x / (1.f + expf(-x)); }
// in bf16 the activation is rounded like the projection it follows
__device__ __forceinline__ float silu(float x, bf16*) { return __bfloat162float(__float2bfloat16(x / (1.f + __expf(-x)))); }
template <typename T>
__device__ __forceinline__ float activate(float x, int act) { return act ? silu(x, static_cast<T*>(nullptr)) : x; }

constexpr int THREADS = 256, WARPS = 8;

// grid (H, value tiles, rows).  A thread owns V value columns of the key rows `group`, `group + GROUPS`, ...; LANES threads cover a tile.
template <typename T, int V, int LANES>
__global__ void __launch_bounds__(THREADS)
decayed_step_kernel(const T* __restrict__ qkv, const float* __restrict__ decay, float* __restrict__ state, const int* __restrict__ positions,
                    const int* __restrict__ row_ids, int H, int dk, int dv, int act, T* __restrict__ out) {
  constexpr int GROUPS = THREADS / LANES, TILE = LANES * V, UNROLL = 8;
  extern __shared__ float sm[];                 // q [dk], k [dk], partial [GROUPS][TILE]
  float* sq = sm;
  float* sk = sq + dk;
  float* part = sk + dk;
  const int h = blockIdx.x, row = blockIdx.z;
  const int pos = positions[row];
  const int lane = threadIdx.x % LANES, group = threadIdx.x / LANES;
  const int col = blockIdx.y * TILE + lane * V;
  T* o = out + (static_cast<long long>(row) * H + h) * dv;
  if (pos < 0) {
    if (group == 0)
      for (int j = 0; j < V; ++j) if (col + j < dv) st(o + col + j, 0.f);
    return;
  }
  const T* base = qkv + static_cast<long long>(row) * H * (2 * dk + dv);
  for (int i = threadIdx.x; i < dk; i += THREADS) {
    sq[i] = activate<T>(ld(base + h * dk + i), act);
    sk[i] = activate<T>(ld(base + (H + h) * dk + i), act);
  }
  const bool live = col < dv;                   // V divides dv where V > 1
  float v[V], acc[V];
#pragma unroll
  for (int j = 0; j < V; ++j) { acc[j] = 0.f; v[j] = live ? activate<T>(ld(base + 2 * H * dk + h * dv + col + j), act) : 0.f; }
  const int r = row_ids == nullptr ? row : row_ids[row];
  float* S = state + (static_cast<long long>(r) * H + h) * dk * dv;
  const float a = decay[h];
  const bool fresh = pos == 0;
  __syncthreads();
  for (int k0 = group; k0 < dk; k0 += GROUPS * UNROLL) {
    float x[UNROLL][V];
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
      const int k = k0 + u * GROUPS;
#pragma unroll
      for (int j = 0; j < V; ++j) x[u][j] = 0.f;
      if (live && k < dk && !fresh) {
        if constexpr (V == 4) {
          const float4 f = *reinterpret_cast<const float4*>(S + static_cast<long long>(k) * dv + col);
          x[u][0] = f.x; x[u][1] = f.y; x[u][2] = f.z; x[u][3] = f.w;
        } else {
          x[u][0] = S[static_cast<long long>(k) * dv + col];
        }
      }
    }
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
      const int k = k0 + u * GROUPS;
      if (live && k < dk) {
        const float kk = sk[k], qq = sq[k];
#pragma unroll
        for (int j = 0; j < V; ++j) { x[u][j] = a * x[u][j] + kk * v[j]; acc[j] += x[u][j] * qq; }
        if constexpr (V == 4) *reinterpret_cast<float4*>(S + static_cast<long long>(k) * dv + col) = make_float4(x[u][0], x[u][1], x[u][2], x[u][3]);
        else S[static_cast<long long>(k) * dv + col] = x[u][0];
      }
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) part[group * TILE + lane * V + j] = acc[j];
  __syncthreads();
  for (int c = threadIdx.x; c < TILE; c += THREADS) {
    float s = 0.f;
#pragma unroll
    for (int g = 0; g < GROUPS; ++g) s += part[g * TILE + c];
    const int cc = blockIdx.y * TILE + c;
    if (cc < dv) st(o + cc, s);
  }
}

// grid (H, ceil(dv / 32), rows).  Lane = value column, warp = a slice of the key rows; the state slice stays in registers over the call.
constexpr int CHUNK = 32;
template <typename T, int KR>
__global__ void __launch_bounds__(THREADS)
decayed_sequence_kernel(const T* __restrict__ qkv, const float* __restrict__ decay, float* __restrict__ state, const int* __restrict__ positions,
                        const int* __restrict__ row_ids, int S_len, int H, int dk, int dv, int act, T* __restrict__ out) {
  extern __shared__ __align__(16) float sm[];
  constexpr int DK = KR * WARPS;
  float* sq = sm;                               // [CHUNK][DK]
  float* sk = sq + CHUNK * DK;                  // [CHUNK][DK]
  float* sv = sk + CHUNK * DK;                  // [CHUNK][32]
  float* part = sv + CHUNK * 32;                // [CHUNK][WARPS][32]
  const int h = blockIdx.x, row = blockIdx.z, c0 = blockIdx.y * 32;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int col = c0 + lane, k0 = warp * KR;
  const int* pos = positions + static_cast<long long>(row) * S_len;
  const long long width = static_cast<long long>(H) * (2 * dk + dv);
  const T* base = qkv + static_cast<long long>(row) * S_len * width;
  T* o = out + (static_cast<long long>(row) * S_len * H + h) * dv;
  const int r = row_ids == nullptr ? row : row_ids[row];
  float* S = state == nullptr ? nullptr : state + (static_cast<long long>(r) * H + h) * dk * dv;
  const float a = decay[h];
  float x[KR];
  const bool load_state = S != nullptr && pos[0] > 0;
#pragma unroll
  for (int i = 0; i < KR; ++i) x[i] = (load_state && k0 + i < dk && col < dv) ? S[static_cast<long long>(k0 + i) * dv + col] : 0.f;
  for (int t0 = 0; t0 < S_len; t0 += CHUNK) {
    const int n = min(CHUNK, S_len - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < n * DK; i += THREADS) {
      const int t = i / DK, c = i - t * DK;
      const T* p = base + (t0 + t) * width;
      sq[i] = c < dk ? activate<T>(ld(p + h * dk + c), act) : 0.f;
      sk[i] = c < dk ? activate<T>(ld(p + (H + h) * dk + c), act) : 0.f;
    }
    for (int i = threadIdx.x; i < n * 32; i += THREADS) {
      const int t = i >> 5, c = c0 + (i & 31);
      sv[i] = c < dv ? activate<T>(ld(base + (t0 + t) * width + 2 * H * dk + h * dv + c), act) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      float acc = 0.f;
      if (pos[t0 + t] >= 0) {
        const float v = sv[t * 32 + lane];
#pragma unroll
        for (int i = 0; i < KR; i += 4) {
          const float4 kk = *reinterpret_cast<const float4*>(sk + t * DK + k0 + i);
          const float4 qq = *reinterpret_cast<const float4*>(sq + t * DK + k0 + i);
          x[i] = a * x[i] + kk.x * v;             acc += x[i] * qq.x;
          x[i + 1] = a * x[i + 1] + kk.y * v;     acc += x[i + 1] * qq.y;
          x[i + 2] = a * x[i + 2] + kk.z * v;     acc += x[i + 2] * qq.z;
          x[i + 3] = a * x[i + 3] + kk.w * v;     acc += x[i + 3] * qq.w;
        }
      }
      part[(t * WARPS + warp) * 32 + lane] = acc;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * 32; i += THREADS) {
      const int t = i >> 5, c = i & 31;
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < WARPS; ++w) s += part[(t * WARPS + w) * 32 + c];
      if (c0 + c < dv) st(o + (t0 + t) * static_cast<long long>(H) * dv + c0 + c, s);
    }
  }
  if (S != nullptr && pos[0] >= 0) {
#pragma unroll
    for (int i = 0; i < KR; ++i)
      if (k0 + i < dk && col < dv) S[static_cast<long long>(k0 + i) * dv + col] = x[i];
  }
}

// Chunked form.  Within a chunk starting from state S:
//     o_i = a^{i+1} S^T q_i + sum_{j <= i} a^{i-j} (q_i . k_j) v_j,      S' = a^n S + sum_j a^{n-1-j} k_j v_j^T
// grid (H, ceil(dv / 64), rows), 8 warps.  The fp32 state lives in accumulator registers for the whole call.  Every factor that is not a
// bf16 activation - the state, the decayed scores, the decayed keys - enters its product as a pair of bf16 (value and rounding rest), so the
// products see 16 bits of it.  The next chunk's rows are fetched into registers while this one is computed.
constexpr int CT = 64, VT = 64;       // tokens per chunk, value columns per CTA

template <int DK>
struct ChunkSmem {
  bf16 q[CT][DK + 8], k[CT][DK + 8], v[CT][VT + 8];
  bf16 s_big[DK][VT + 8], s_rest[DK][VT + 8];
  float pw[CT + 1];
  int count;
};

template <int DK>
__global__ void __launch_bounds__(THREADS, 2)
decayed_chunks_kernel(const bf16* __restrict__ qkv, const float* __restrict__ decay, float* __restrict__ state, const int* __restrict__ positions,
                      const int* __restrict__ row_ids, int S_len, int H, int dk, int dv, int act, bf16* __restrict__ out) {
  using namespace mma16;
  extern __shared__ __align__(16) uint8_t raw[];
  ChunkSmem<DK>& sm = *reinterpret_cast<ChunkSmem<DK>*>(raw);
  constexpr int MT = DK / 16;                      // 16-row tiles of the state: 8 (a warp each, all columns) or 4 (two warps each, half the columns)
  constexpr int NT = MT;                           // 8-column tiles of the state a warp owns
  constexpr int QV = DK / 8 * CT / THREADS, VV = VT / 8 * CT / THREADS;
  const int h = blockIdx.x, row = blockIdx.z, c0 = blockIdx.y * VT;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int* pos = positions + static_cast<long long>(row) * S_len;
  const long long width = static_cast<long long>(H) * (2 * dk + dv);
  const bf16* base = qkv + static_cast<long long>(row) * S_len * width;
  bf16* o = out + (static_cast<long long>(row) * S_len * H + h) * dv;
  const float a = decay[h];
  if (tid == 0) sm.count = 0;
  for (int i = tid; i <= CT; i += THREADS) sm.pw[i] = powf(a, static_cast<float>(i));
  __syncthreads();
  {
    int live = 0;
    for (int i = tid; i < S_len; i += THREADS) live += pos[i] >= 0;
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) live += __shfl_xor_sync(0xffffffffu, live, s);
    if (lane == 0) atomicAdd(&sm.count, live);
  }
  __syncthreads();
  const int len = sm.count;                        // positions below 0 come last
  const int r = row_ids == nullptr ? row : row_ids[row];
  float* S = state == nullptr ? nullptr : state + (static_cast<long long>(r) * H + h) * dk * dv;
  const int g = lane >> 2, t2 = (lane & 3) * 2;
  // this warp's part of the state: rows sm_row + {g, g + 8}, columns s_col + 8 n + t2 + {0, 1}
  const int s_row = (MT == 8 ? warp : warp & 3) * 16, s_col = MT == 8 ? 0 : (warp >> 2) * 32;
  float st_acc[NT][4];
  const bool load_state = S != nullptr && len > 0 && pos[0] > 0;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int kr = s_row + g + (e >> 1) * 8, vc = c0 + s_col + n * 8 + t2 + (e & 1);
      st_acc[n][e] = (load_state && kr < dk && vc < dv) ? S[static_cast<long long>(kr) * dv + vc] : 0.f;
    }
  // output tile of this warp: tokens o_row + {g, g + 8}, columns o_col + ...
  const int o_row = (warp & 3) * 16, o_col = (warp >> 2) * 32;
  uint4 rq[QV], rk[QV], rv[VV];
  const uint4 zero = make_uint4(0, 0, 0, 0);
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < QV; ++i) {
      const int x = tid + i * THREADS, t = x / (DK / 8), c = (x % (DK / 8)) * 8;
      const bool ok = t0 + t < len && c < dk;
      const bf16* p = base + (t0 + t) * width + h * dk + c;
      rq[i] = ok ? *reinterpret_cast<const uint4*>(p) : zero;
      rk[i] = ok ? *reinterpret_cast<const uint4*>(p + H * dk) : zero;
    }
#pragma unroll
    for (int i = 0; i < VV; ++i) {
      const int x = tid + i * THREADS, t = x / (VT / 8), c = (x % (VT / 8)) * 8;
      rv[i] = t0 + t < len && c0 + c < dv ? *reinterpret_cast<const uint4*>(base + (t0 + t) * width + 2 * H * dk + h * dv + c0 + c) : zero;
    }
  };
  auto put = [&](bf16* dst, uint4 x) {
    if (act) {
      uint32_t w[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float f0 = lo_f(w[j]), f1 = hi_f(w[j]);
        w[j] = pack2(__fdividef(f0, 1.f + __expf(-f0)), __fdividef(f1, 1.f + __expf(-f1)));
      }
      x = make_uint4(w[0], w[1], w[2], w[3]);
    }
    *reinterpret_cast<uint4*>(dst) = x;
  };
  fetch(0);
  for (int t0 = 0; t0 < len; t0 += CT) {
    const int n = min(CT, len - t0);
    __syncthreads();                               // the chunk before has been read
#pragma unroll
    for (int i = 0; i < QV; ++i) {
      const int x = tid + i * THREADS, t = x / (DK / 8), c = (x % (DK / 8)) * 8;
      put(&sm.q[t][c], rq[i]);
      put(&sm.k[t][c], rk[i]);
    }
#pragma unroll
    for (int i = 0; i < VV; ++i) {
      const int x = tid + i * THREADS, t = x / (VT / 8), c = (x % (VT / 8)) * 8;
      put(&sm.v[t][c], rv[i]);
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t big, rest;
        split2(st_acc[j][2 * e], st_acc[j][2 * e + 1], big, rest);
        *reinterpret_cast<uint32_t*>(&sm.s_big[s_row + g + 8 * e][s_col + j * 8 + t2]) = big;
        *reinterpret_cast<uint32_t*>(&sm.s_rest[s_row + g + 8 * e][s_col + j * 8 + t2]) = rest;
      }
    __syncthreads();
    if (t0 + CT < len) fetch(t0 + CT);
    // ---- from the state: Q S
    float acc[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) { acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f; }
#pragma unroll
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t qa[4];
      ldsm4(qa, smem_addr(&sm.q[o_row + (lane & 15)][kk + (lane >> 4) * 8]));
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        uint32_t b[4], d[4];
        ldsm4_t(b, smem_addr(&sm.s_big[kk + (lane & 15)][o_col + j * 16 + (lane >> 4) * 8]));
        ldsm4_t(d, smem_addr(&sm.s_rest[kk + (lane & 15)][o_col + j * 16 + (lane >> 4) * 8]));
        mma(acc[2 * j], qa, b[0], b[1]);
        mma(acc[2 * j + 1], qa, b[2], b[3]);
        mma(acc[2 * j], qa, d[0], d[1]);
        mma(acc[2 * j + 1], qa, d[2], d[3]);
      }
    }
    const float w0 = sm.pw[o_row + g + 1], w1 = sm.pw[o_row + g + 9];
#pragma unroll
    for (int j = 0; j < 4; ++j) { acc[j][0] *= w0; acc[j][1] *= w0; acc[j][2] *= w1; acc[j][3] *= w1; }
    // ---- from the chunk: 16 tokens at a time, up to this warp's diagonal tile
#pragma unroll 1
    for (int j = 0; j <= (warp & 3); ++j) {
      float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
      for (int kk = 0; kk < DK; kk += 16) {
        uint32_t qa[4], b[4];
        ldsm4(qa, smem_addr(&sm.q[o_row + (lane & 15)][kk + (lane >> 4) * 8]));
        ldsm4(b, smem_addr(&sm.k[j * 16 + (lane & 7) + (lane >> 4) * 8][kk + ((lane >> 3) & 1) * 8]));
        mma(sc[0], qa, b[0], b[1]);
        mma(sc[1], qa, b[2], b[3]);
      }
      uint32_t pa[4], pr[4];
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = o_row + g + 8 * e, c = j * 16 + half * 8 + t2;
          const float x0 = c <= i ? sc[half][2 * e] * sm.pw[max(i - c, 0)] : 0.f;
          const float x1 = c + 1 <= i ? sc[half][2 * e + 1] * sm.pw[max(i - c - 1, 0)] : 0.f;
          split2(x0, x1, pa[half * 2 + e], pr[half * 2 + e]);
        }
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        uint32_t b[4];
        ldsm4_t(b, smem_addr(&sm.v[j * 16 + (lane & 15)][o_col + m * 16 + (lane >> 4) * 8]));
        mma(acc[2 * m], pa, b[0], b[1]);
        mma(acc[2 * m + 1], pa, b[2], b[3]);
        mma(acc[2 * m], pr, b[0], b[1]);
        mma(acc[2 * m + 1], pr, b[2], b[3]);
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = o_row + g + 8 * e, c = c0 + o_col + j * 8 + t2;
        if (t < n && c < dv) *reinterpret_cast<uint32_t*>(o + (t0 + t) * static_cast<long long>(H) * dv + c) = pack2(acc[j][2 * e], acc[j][2 * e + 1]);
      }
    // ---- the state after the chunk
    const float wn = sm.pw[n];
#pragma unroll
    for (int j = 0; j < NT; ++j) { st_acc[j][0] *= wn; st_acc[j][1] *= wn; st_acc[j][2] *= wn; st_acc[j][3] *= wn; }
#pragma unroll
    for (int kt = 0; kt < CT; kt += 16) {
      if (kt < n) {
        uint32_t ka[4], big[4], rest[4];
        // A = K^T: rows are key components, the reduction runs over tokens
        ldsm4_t(ka, smem_addr(&sm.k[kt + (lane & 7) + (lane >> 4) * 8][s_row + ((lane >> 3) & 1) * 8]));
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int tk = kt + (x >> 1) * 8 + t2;   // tokens past the end carry zero keys
          split2(lo_f(ka[x]) * sm.pw[max(n - 1 - tk, 0)], hi_f(ka[x]) * sm.pw[max(n - 2 - tk, 0)], big[x], rest[x]);
        }
#pragma unroll
        for (int m = 0; m < NT / 2; ++m) {
          uint32_t b[4];
          ldsm4_t(b, smem_addr(&sm.v[kt + (lane & 15)][s_col + m * 16 + (lane >> 4) * 8]));
          mma(st_acc[2 * m], big, b[0], b[1]);
          mma(st_acc[2 * m + 1], big, b[2], b[3]);
          mma(st_acc[2 * m], rest, b[0], b[1]);
          mma(st_acc[2 * m + 1], rest, b[2], b[3]);
        }
      }
    }
  }
  if (S != nullptr && len > 0) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int kr = s_row + g + (e >> 1) * 8, vc = c0 + s_col + n * 8 + t2 + (e & 1);
        if (kr < dk && vc < dv) S[static_cast<long long>(kr) * dv + vc] = st_acc[n][e];
      }
  }
  for (int i = tid; i < (S_len - len) * (VT / 8); i += THREADS) {
    const int t = len + i / (VT / 8), c = c0 + (i % (VT / 8)) * 8;
    if (c < dv) *reinterpret_cast<uint4*>(o + t * static_cast<long long>(H) * dv + c) = zero;
  }
}

template <typename T, int V, int LANES>
int step_go(const T* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int H, int dk, int dv, int act, T* out,
            cudaStream_t stream) {
  const int tile = LANES * V;
  const size_t smem = static_cast<size_t>(2 * dk + THREADS * V) * 4;
  if (smem > 200 * 1024) return -3;
  cudaError_t e = cudaFuncSetAttribute(decayed_step_kernel<T, V, LANES>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  decayed_step_kernel<T, V, LANES><<<dim3(H, (dv + tile - 1) / tile, R), THREADS, smem, stream>>>(qkv, decay, state, positions, row_ids, H, dk, dv, act, out);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int step_any(const T* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int H, int dk, int dv, int act, T* out,
             cudaStream_t stream) {
  if (dv % 4 != 0 || (reinterpret_cast<uintptr_t>(state) & 15)) return step_go<T, 1, 32>(qkv, decay, state, positions, row_ids, R, H, dk, dv, act, out, stream);
  // narrow tiles while there are few (row, head) pairs, so that every SM has state to move
  if (static_cast<long long>(R) * H < 592 || dv <= 32) return step_go<T, 4, 8>(qkv, decay, state, positions, row_ids, R, H, dk, dv, act, out, stream);
  return step_go<T, 4, 32>(qkv, decay, state, positions, row_ids, R, H, dk, dv, act, out, stream);
}

template <typename T, int KR>
int seq_go(const T* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int S, int H, int dk, int dv, int act,
           T* out, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(2 * CHUNK * KR * WARPS + CHUNK * 32 + CHUNK * WARPS * 32) * 4;
  cudaError_t e = cudaFuncSetAttribute(decayed_sequence_kernel<T, KR>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  decayed_sequence_kernel<T, KR><<<dim3(H, (dv + 31) / 32, R), THREADS, smem, stream>>>(qkv, decay, state, positions, row_ids, S, H, dk, dv, act, out);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int seq_any(const T* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int S, int H, int dk, int dv, int act,
            T* out, cudaStream_t stream) {
#define DEWB_SEQ(KK) seq_go<T, KK>(qkv, decay, state, positions, row_ids, R, S, H, dk, dv, act, out, stream)
  if (dk <= 32) return DEWB_SEQ(4);
  if (dk <= 64) return DEWB_SEQ(8);
  if (dk <= 128) return DEWB_SEQ(16);
  if (dk <= 256) return DEWB_SEQ(32);
  if (dk <= 512) return DEWB_SEQ(64);
#undef DEWB_SEQ
  return -3;
}

template <int DK>
int chunks_go(const bf16* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int S, int H, int dk, int dv, int act,
              bf16* out, cudaStream_t stream) {
  const int smem = static_cast<int>(sizeof(ChunkSmem<DK>));
  cudaError_t e = cudaFuncSetAttribute(decayed_chunks_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  decayed_chunks_kernel<DK><<<dim3(H, (dv + VT - 1) / VT, R), THREADS, smem, stream>>>(qkv, decay, state, positions, row_ids, S, H, dk, dv, act, out);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace decayed
}  // namespace dewb

using namespace dewb::decayed;

// One token per row: qkv [R, H (2 dk + dv)], positions [R], out [R, H, dv].
extern "C" int dewb_decayed_step(const void* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int H, int dk,
                                 int dv, int act, void* out, int fp32, void* stream_ptr) {
  if (R <= 0) return 0;
  if (H < 1 || dk < 1 || dv < 1 || state == nullptr) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (fp32) return step_any<float>(static_cast<const float*>(qkv), decay, state, positions, row_ids, R, H, dk, dv, act, static_cast<float*>(out), stream);
  return step_any<bf16>(static_cast<const bf16*>(qkv), decay, state, positions, row_ids, R, H, dk, dv, act, static_cast<bf16*>(out), stream);
}

// qkv [R, S, H (2 dk + dv)], positions [R, S], out [R, S, H, dv]; `state` may be null (start from zero, keep nothing).
extern "C" int dewb_decayed_sequence(const void* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int S, int H,
                                     int dk, int dv, int act, void* out, int fp32, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (H < 1 || dk < 1 || dv < 1) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (fp32) return seq_any<float>(static_cast<const float*>(qkv), decay, state, positions, row_ids, R, S, H, dk, dv, act, static_cast<float*>(out), stream);
  return seq_any<bf16>(static_cast<const bf16*>(qkv), decay, state, positions, row_ids, R, S, H, dk, dv, act, static_cast<bf16*>(out), stream);
}

// The chunked tensor-core form of the same (bf16; dk, dv multiples of 8, dk at most 128; qkv and out on 16-byte boundaries).
extern "C" int dewb_decayed_chunks(const void* qkv, const float* decay, float* state, const int* positions, const int* row_ids, int R, int S, int H,
                                   int dk, int dv, int act, void* out, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (H < 1 || dk < 8 || dv < 8 || dk % 8 || dv % 8 || dk > 128 || (reinterpret_cast<uintptr_t>(qkv) & 15) || (reinterpret_cast<uintptr_t>(out) & 15)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bf16* x = static_cast<const bf16*>(qkv);
  if (dk <= 64) return chunks_go<64>(x, decay, state, positions, row_ids, R, S, H, dk, dv, act, static_cast<bf16*>(out), stream);
  return chunks_go<128>(x, decay, state, positions, row_ids, R, S, H, dk, dv, act, static_cast<bf16*>(out), stream);
}
