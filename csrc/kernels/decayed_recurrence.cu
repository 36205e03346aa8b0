// Linear attention with a constant decay per head (lightning attention), for sm_100a:
//     S_t = decay S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t,   q, k, v = silu of the packed projection (or as given)
//
//   decayed_step        one token per row: the fp32 state is read and written once
//   decayed_sequence    a call's tokens one after another, any head widths, fp32 arithmetic (the exact form; it also serves fp32 models)
//
// The packed projection is [rows, S, H dk | H dk | H dv] (q, k, v; heads inside each).  `state` [store rows, H, dk, dv] fp32 stays on the
// device between calls; a call row whose first position is 0 starts from zero, positions below 0 are padding (they come last in a row,
// change no state and give zero outputs).  Compiled without fast math.
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

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
