// Mixture-of-experts feed-forward outside training, on one rank, for sm_100a: no statistics, no saved state, no host synchronisation.
//
//   moe_router    one block per token: the router's logits (fp32 sums of the row with every expert's weight row) and the selection
//   moe_select    the selection alone, one warp per token, from logits another product made (prompts: a tensor-core product)
//   moe_gather    rows sorted by expert, each expert's rows starting on a multiple of 128 (what the tcgen05 grouped product walks), and the
//                 shared expert's gate on the way through the row
//   moe_gemm      the grouped product on the CUDA cores: fp32 models, and sizes the tensor-core kernel does not take
//   moe_glu       silu(gate) * up on the rows in use
//   moe_combine   a token's rows times their weights, plus the shared expert's output times its gate, in fp32
//
// Selection: logits may carry a bias; scores are a sigmoid or softmax of the logits, or the logits themselves, whose weights are then the softmax over
// the chosen ones alone; choice scores add a bias that steers the choice only; with groups, a group counts
// the sum of its two best choice scores (or its best one) and the experts outside a token's best groups are out of the choice (their choice scores become
// `fill`); the weights are the chosen scores, divided by their sum where `norm` asks for it.  Tokens at positions below 0 are padding: no
// expert runs for them.  A row's place among its expert's rows comes from an atomic counter, so it may differ from run to run; the rows of a
// product do not depend on each other.  Compiled without fast math.
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/rows.cuh"

namespace dewb {
namespace moeserve {

using namespace rows;

constexpr uint32_t FULL = 0xffffffffu;
constexpr int THREADS = 256, WARPS = THREADS / 32;
constexpr int MAX_E = 1024, MAX_K = 32, BLOCK = 128;

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(FULL, v, o);
  return v;
}
__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }

struct Choice {
  const float* bias;       // [E] or null: steers the choice alone
  const float* logit_bias;  // [E] or null: part of the logits
  int E, k, groups, keep, best;   // a group counts the sum of its `best` (1 or 2) best choice scores
  float fill;              // choice score of experts outside the kept groups
  int score, norm;         // score 0: softmax, 1: sigmoid, 2: the logits, weights by the softmax over the chosen ones
  float scaling;
  float* weights;          // [T, k]
  int* ids;                // [T, k], -1: padding
  int* rank;               // [T, k] place among the expert's rows
  int* counts;             // [E]
};

// One warp: sc holds the token's logits (expert lane + 32 i); s_sel [E] and s_group [groups] are the warp's own shared memory.
template <int NI>
__device__ __forceinline__ void choose(const Choice& c, long long t, bool live, float (&sc)[NI], float* s_sel, float* s_group) {
  const int lane = threadIdx.x & 31;
  if (!live) {
    if (lane < c.k) { c.weights[t * c.k + lane] = 0.f; c.ids[t * c.k + lane] = -1; }
    return;
  }
  if (c.logit_bias != nullptr) {
#pragma unroll
    for (int i = 0; i < NI; ++i) if (lane + 32 * i < c.E) sc[i] += c.logit_bias[lane + 32 * i];
  }
  if (c.score == 1) {
#pragma unroll
    for (int i = 0; i < NI; ++i) sc[i] = sigmoid(sc[i]);
  } else if (c.score == 0) {
    float mx = -INFINITY, sum = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) if (lane + 32 * i < c.E) mx = fmaxf(mx, sc[i]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(FULL, mx, o));
#pragma unroll
    for (int i = 0; i < NI; ++i) { sc[i] = lane + 32 * i < c.E ? expf(sc[i] - mx) : 0.f; sum += sc[i]; }
    sum = warp_sum(sum);
#pragma unroll
    for (int i = 0; i < NI; ++i) sc[i] /= sum;
  }
  float sel[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int e = lane + 32 * i;
    sel[i] = e < c.E ? sc[i] + (c.bias != nullptr ? c.bias[e] : 0.f) : -INFINITY;
  }
  if (c.groups > 1) {
    const int per = c.E / c.groups;
#pragma unroll
    for (int i = 0; i < NI; ++i) if (lane + 32 * i < c.E) s_sel[lane + 32 * i] = sel[i];
    __syncwarp();
    for (int g = lane; g < c.groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;             // the group's best and second best
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float v = s_sel[e];
        if (v > a) { b = a; a = v; } else if (v > b) b = v;
      }
      s_group[g] = per > 1 && c.best > 1 ? a + b : a;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = lane + 32 * i;
      if (e < c.E) {
        const int g = e / per;
        int before = 0;
        for (int o = 0; o < c.groups; ++o) before += s_group[o] > s_group[g] || (s_group[o] == s_group[g] && o < g);
        if (before >= c.keep) sel[i] = c.fill;
      }
    }
    __syncwarp();                                     // s_sel and s_group are the next token's as well
  }
  float my_w = 0.f, wsum = 0.f;
  int my_id = 0;
  for (int j = 0; j < c.k; ++j) {
    float bv = -INFINITY, bs = 0.f;
    int bi = 0x7fffffff;                              // ties go to the lower expert
#pragma unroll
    for (int i = 0; i < NI; ++i)
      if (sel[i] > bv) { bv = sel[i]; bi = lane + 32 * i; bs = sc[i]; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(FULL, bv, o), os = __shfl_xor_sync(FULL, bs, o);
      const int oi = __shfl_xor_sync(FULL, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; bs = os; }
    }
    if (bi >= c.E) bi = j;                            // nothing comparable left (not-a-number logits): stay within the experts
    if ((bi & 31) == lane) {
#pragma unroll
      for (int i = 0; i < NI; ++i) if (i == (bi >> 5)) sel[i] = -INFINITY;
    }
    wsum += bs;
    if (lane == j) { my_w = bs; my_id = bi; }
  }
  if (c.score == 2) {
    float mx = lane < c.k ? my_w : -INFINITY;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(FULL, mx, o));
    my_w = lane < c.k ? expf(my_w - mx) : 0.f;
    my_w /= warp_sum(my_w);
  } else if (c.norm) {
    my_w = my_w / (wsum + 1e-20f);
  }
  if (lane < c.k) {
    c.weights[t * c.k + lane] = my_w * c.scaling;
    c.ids[t * c.k + lane] = my_id;
    c.rank[t * c.k + lane] = atomicAdd(c.counts + my_id, 1);
  }
}

constexpr int SELECT_TOKENS = 32;      // tokens a block selects for: it takes its experts' places with one addition per expert

// logits [T, ld] fp32; `rest` columns further on (0: none) holds what the weights' rounding to bf16 dropped, to be added
template <int NI>
__global__ void __launch_bounds__(THREADS)
moe_select_kernel(const float* __restrict__ logits, long long ld_, int rest, const int* __restrict__ positions, int T, Choice c) {
  extern __shared__ float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s_sel = smem + warp * (c.E + c.groups);
  int* s_count = reinterpret_cast<int*>(smem + WARPS * (c.E + c.groups));
  int* const counts = c.counts;
  for (int e = threadIdx.x; e < c.E; e += THREADS) s_count[e] = 0;
  __syncthreads();
  c.counts = s_count;
  const long long t0 = static_cast<long long>(blockIdx.x) * SELECT_TOKENS, t1 = t0 + SELECT_TOKENS < T ? t0 + SELECT_TOKENS : T;
  for (long long t = t0 + warp; t < t1; t += WARPS) {
    float sc[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = lane + 32 * i;
      sc[i] = e < c.E ? logits[t * ld_ + e] + (rest > 0 ? logits[t * ld_ + rest + e] : 0.f) : 0.f;
    }
    choose<NI>(c, t, positions == nullptr || positions[t] >= 0, sc, s_sel, s_sel + c.E);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < c.E; e += THREADS)
    if (s_count[e] > 0) s_count[e] = atomicAdd(counts + e, s_count[e]);
  __syncthreads();
  for (long long t = t0 + warp; t < t1; t += WARPS)      // the lanes that wrote these places
    if (lane < c.k && c.ids[t * c.k + lane] >= 0) c.rank[t * c.k + lane] += s_count[c.ids[t * c.k + lane]];
}

// x [T, d], w [E, d]
template <typename T, typename W, int V, int NI>
__global__ void __launch_bounds__(THREADS)
moe_router_kernel(const T* __restrict__ x, const W* __restrict__ w, const int* __restrict__ positions, int d, Choice c) {
  extern __shared__ __align__(16) float smem[];
  const int dp = (d + 3) & ~3;
  float *sx = smem, *s_logit = smem + dp, *s_sel = s_logit + c.E;
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool live = positions == nullptr || positions[t] >= 0;
  if (live) {
    for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
      float a[V];
      load_v<V>(x + t * d + i, a);
      store_v<V>(sx + i, a);
    }
    __syncthreads();
    for (int e = warp; e < c.E; e += WARPS) {
      const W* row = w + static_cast<long long>(e) * d;
      float s = 0.f;
#pragma unroll 4
      for (int i = lane * V; i < d; i += 32 * V) {
        float a[V], b[V];
        load_v<V>(sx + i, a);
        load_v<V>(row + i, b);
#pragma unroll
        for (int j = 0; j < V; ++j) s += a[j] * b[j];
      }
      s = warp_sum(s);
      if (lane == 0) s_logit[e] = s;
    }
    __syncthreads();
  }
  if (warp != 0) return;
  float sc[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) sc[i] = live && lane + 32 * i < c.E ? s_logit[lane + 32 * i] : 0.f;
  choose<NI>(c, t, live, sc, s_sel, s_sel + c.E);
}

// Starts of the experts' rows: off[e], off[E] = rows in use (whole blocks of 128).
__device__ void expert_offsets(const int* __restrict__ counts, int E, int* off) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x, per = (E + 31) / 32, e0 = min(E, lane * per), e1 = min(E, e0 + per);
    int sum = 0;
    for (int e = e0; e < e1; ++e) sum += (counts[e] + BLOCK - 1) / BLOCK * BLOCK;
    int incl = sum;
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(FULL, incl, o);
      if (lane >= o) incl += v;
    }
    int run = incl - sum;
    for (int e = e0; e < e1; ++e) { off[e] = run; run += (counts[e] + BLOCK - 1) / BLOCK * BLOCK; }
    if (lane == 31) off[E] = incl;
  }
  __syncthreads();
}

// x [T, d] -> rows [rows_cap, d]; place [T, k] (-1: padding); tile_group [rows_cap / 128]; offsets [E + 1]; with `gate_w` [d] also
// gate [T] = sigmoid(gate_w . x)
template <typename T, int V>
__global__ void __launch_bounds__(THREADS)
moe_gather_kernel(const T* __restrict__ x, const int* __restrict__ ids, const int* __restrict__ rank, const int* __restrict__ counts,
                  const T* __restrict__ gate_w, T* __restrict__ rows_out, int* __restrict__ place, int* __restrict__ tile_group,
                  int* __restrict__ offsets, float* __restrict__ gate, int tokens, int d, int E, int k, int tiles) {
  __shared__ int off[MAX_E + 1];
  expert_offsets(counts, E, off);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e <= E; e += THREADS) offsets[e] = off[e];
    for (int tl = threadIdx.x; tl < tiles; tl += THREADS) {
      const int start = tl * BLOCK;
      int g = -1;
      if (start < off[E]) {
        int lo = 0, hi = E;                           // the last expert that starts at or before the tile (empty ones share a start)
        while (hi - lo > 1) {
          const int mid = (lo + hi) >> 1;
          if (off[mid] <= start) lo = mid; else hi = mid;
        }
        g = lo;
      }
      tile_group[tl] = g;
    }
  }
  const int cap = tiles * BLOCK;
  for (long long t = static_cast<long long>(blockIdx.x) * WARPS + warp; t < tokens; t += static_cast<long long>(gridDim.x) * WARPS) {
    int my = -1;
    if (lane < k) {
      const int e = ids[t * k + lane];
      if (e >= 0) my = off[e] + rank[t * k + lane];
      if (my >= cap) my = -1;                         // cannot happen: the buffer holds every pair
      place[t * k + lane] = my;
    }
    float dot = 0.f;
    const int top = (d + 32 * V - 1) / (32 * V) * (32 * V);        // every lane stays for the shuffles
    for (int i = lane * V; i < top; i += 32 * V) {
      float a[V];
      if (i < d) {
        load_v<V>(x + t * d + i, a);
        if (gate_w != nullptr) {
          float b[V];
          load_v<V>(gate_w + i, b);
#pragma unroll
          for (int j = 0; j < V; ++j) dot += a[j] * b[j];
        }
      }
      for (int j = 0; j < k; ++j) {
        const int p = __shfl_sync(FULL, my, j);
        if (p >= 0 && i < d) store_v<V>(rows_out + static_cast<long long>(p) * d + i, a);
      }
    }
    if (gate_w != nullptr) {
      dot = warp_sum(dot);
      if (lane == 0) gate[t] = sigmoid(dot);
    }
  }
}

// out [rows, N] = a [rows, K] w[expert of the row]^T, w [E, N, K]: 64 x 64 tiles, 4 x 4 sums a thread
template <typename T>
__global__ void __launch_bounds__(THREADS)
moe_gemm_kernel(const T* __restrict__ a, const T* __restrict__ w, T* __restrict__ out, const int* __restrict__ tile_group,
                const int* __restrict__ offsets, const int* __restrict__ counts, int N, int K) {
  constexpr int M = 64, NT = 64, KT = 16;
  __shared__ __align__(16) float sa[KT][M + 4], sw[KT][NT + 4];
  const int r0 = blockIdx.y * M, n0 = blockIdx.x * NT;
  const int g = tile_group[r0 / BLOCK];
  if (g < 0) return;
  const int end = offsets[g] + counts[g];
  if (r0 >= end) return;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += KT) {
    for (int i = threadIdx.x; i < M * KT; i += THREADS) {
      const int r = i / KT, c = i - r * KT;
      sa[c][r] = r0 + r < end && k0 + c < K ? ld(a + static_cast<long long>(r0 + r) * K + k0 + c) : 0.f;
      sw[c][r] = n0 + r < N && k0 + c < K ? ld(w + (static_cast<long long>(g) * N + n0 + r) * K + k0 + c) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < KT; ++c) {
      const float4 x4 = *reinterpret_cast<const float4*>(&sa[c][ty * 4]), y4 = *reinterpret_cast<const float4*>(&sw[c][tx * 4]);
      const float x[4] = {x4.x, x4.y, x4.z, x4.w}, y[4] = {y4.x, y4.y, y4.z, y4.w};
#pragma unroll
      for (int p = 0; p < 4; ++p)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[p][q] += x[p] * y[q];
    }
    __syncthreads();
  }
#pragma unroll
  for (int p = 0; p < 4; ++p) {
    const int r = r0 + ty * 4 + p;
    if (r >= end) continue;
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int n = n0 + tx * 4 + q;
      if (n >= N) continue;
      const float v[1] = {acc[p][q]};
      store_v<1>(out + static_cast<long long>(r) * N + n, v);
    }
  }
}

// x sigmoid(x): fp32 models take the exact quotient, bf16 the approximate one (a few parts in 2^22)
template <typename T>
__device__ __forceinline__ float silu(float x) {
  if constexpr (sizeof(T) == 2) return __fdividef(x, 1.f + __expf(-x));
  else return x / (1.f + expf(-x));
}

// gu [rows, 2 F] -> out [rows, F], a warp a row
template <typename T, int V>
__global__ void __launch_bounds__(THREADS)
moe_glu_kernel(const T* __restrict__ gu, T* __restrict__ out, const int* __restrict__ tile_group, const int* __restrict__ offsets,
               const int* __restrict__ counts, int F) {
  const int r = blockIdx.x * WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int g = tile_group[r / BLOCK];
  if (g < 0 || r >= offsets[g] + counts[g]) return;
  const T* src = gu + static_cast<long long>(r) * 2 * F;
  for (int i = lane * V; i < F; i += 32 * V) {
    float a[V], b[V];
    load_v<V>(src + i, a);
    load_v<V>(src + F + i, b);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = silu<T>(a[j]) * b[j];
    store_v<V>(out + static_cast<long long>(r) * F + i, a);
  }
}

constexpr int COMBINE = 128;

// grid (tokens, ceil(d / (COMBINE V))); shared [T, d] with gate [T] fp32 (null gate: 1), or null
template <typename T, int V>
__global__ void __launch_bounds__(COMBINE)
moe_combine_kernel(const T* __restrict__ y, const float* __restrict__ weights, const int* __restrict__ place, const T* __restrict__ shared,
                   const float* __restrict__ gate, T* __restrict__ out, int d, int k) {
  __shared__ float s_w[MAX_K];
  __shared__ int s_p[MAX_K];
  const long long t = blockIdx.x;
  if (threadIdx.x < k) { s_w[threadIdx.x] = weights[t * k + threadIdx.x]; s_p[threadIdx.x] = place[t * k + threadIdx.x]; }
  __syncthreads();
  const int i = (blockIdx.y * COMBINE + threadIdx.x) * V;
  if (i >= d) return;
  float acc[V];
#pragma unroll
  for (int j = 0; j < V; ++j) acc[j] = 0.f;
#pragma unroll 4
  for (int q = 0; q < k; ++q) {
    const int p = s_p[q];
    if (p < 0) continue;
    float a[V];
    load_v<V>(y + static_cast<long long>(p) * d + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) acc[j] += s_w[q] * a[j];
  }
  if (shared != nullptr) {
    float a[V];
    load_v<V>(shared + t * d + i, a);
    const float g = gate == nullptr ? 1.f : gate[t];
#pragma unroll
    for (int j = 0; j < V; ++j) acc[j] += g * a[j];
  }
  store_v<V>(out + t * d + i, acc);
}

bool choice_ok(const Choice& c) {
  return c.score >= 0 && c.score <= 2 && c.E >= 1 && c.E <= MAX_E && c.k >= 1 && c.k <= MAX_K && c.k <= c.E && c.groups >= 1 && c.E % c.groups == 0 && c.keep >= 1 && c.keep <= c.groups &&
         c.weights != nullptr && c.ids != nullptr && c.rank != nullptr && c.counts != nullptr;
}

template <typename K>
int allow_smem(K kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 220 * 1024) return -3;
  return static_cast<int>(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
}

template <int NI>
int select(const float* logits, long long ld_, int rest, const int* positions, int T, const Choice& c, cudaStream_t stream) {
  const size_t smem = (static_cast<size_t>(WARPS) * (c.E + c.groups) + c.E) * 4;
  const int r = allow_smem(moe_select_kernel<NI>, smem);
  if (r) return r;
  moe_select_kernel<NI><<<(T + SELECT_TOKENS - 1) / SELECT_TOKENS, THREADS, smem, stream>>>(logits, ld_, rest, positions, T, c);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, typename W, int V>
int router(const T* x, const W* w, const int* positions, int tokens, int d, const Choice& c, cudaStream_t stream) {
  const size_t smem = static_cast<size_t>(((d + 3) & ~3) + 2 * c.E + c.groups) * 4;
#define DEWB_ROUTER(NN) do { const int r = allow_smem(moe_router_kernel<T, W, V, NN>, smem); if (r) return r; \
    moe_router_kernel<T, W, V, NN><<<tokens, THREADS, smem, stream>>>(x, w, positions, d, c); } while (0)
  if (c.E <= 128) DEWB_ROUTER(4); else if (c.E <= 256) DEWB_ROUTER(8); else DEWB_ROUTER(32);
#undef DEWB_ROUTER
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int gather(const void* x, const int* ids, const int* rank, const int* counts, const void* gate_w, void* out, int* place, int* tile_group, int* offsets,
           float* gate, int tokens, int d, int E, int k, int tiles, cudaStream_t stream) {
  const bool a16 = aligned(x, 16) && aligned(gate_w, 16) && aligned(out, 16);
  const int v = a16 && sizeof(T) == 2 && d % 8 == 0 ? 8 : a16 && d % 4 == 0 ? 4 : 1;
  int blocks = (tokens + WARPS - 1) / WARPS;
  blocks = blocks < 148 * 8 ? blocks : 148 * 8;
#define DEWB_GATHER(VV) moe_gather_kernel<T, VV><<<blocks, THREADS, 0, stream>>>(static_cast<const T*>(x), ids, rank, counts, static_cast<const T*>(gate_w), \
    static_cast<T*>(out), place, tile_group, offsets, gate, tokens, d, E, k, tiles)
  if constexpr (sizeof(T) == 2) { if (v == 8) DEWB_GATHER(8); else if (v == 4) DEWB_GATHER(4); else DEWB_GATHER(1); }
  else { if (v == 4) DEWB_GATHER(4); else DEWB_GATHER(1); }
#undef DEWB_GATHER
  return static_cast<int>(cudaGetLastError());
}

}  // namespace moeserve
}  // namespace dewb

using namespace dewb::moeserve;

// logits [T, ld] fp32 (plus logits[., rest + e] when rest > 0) -> weights, ids, rank [T, k], counts [E] (zero before the call).
// `positions` [T] or null: below 0 = padding.
extern "C" int dewb_moe_select(const float* logits, long long ld_, int rest, const float* bias, const float* logit_bias, const int* positions, int T,
                               int E, int k, int groups, int keep, int best, float fill, int score, int norm, float scaling, float* weights, int* ids, int* rank, int* counts,
                               void* stream_ptr) {
  if (T <= 0) return 0;
  const Choice c{bias, logit_bias, E, k, groups, keep, best, fill, score, norm, scaling, weights, ids, rank, counts};
  if (!choice_ok(c) || ld_ < E || rest < 0 || (rest > 0 && ld_ < rest + E)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (E <= 128) return select<4>(logits, ld_, rest, positions, T, c, stream);
  if (E <= 256) return select<8>(logits, ld_, rest, positions, T, c, stream);
  return select<32>(logits, ld_, rest, positions, T, c, stream);
}

// The same with the logits made here: x [T, d] (fp32 or bf16), w [E, d] (fp32, or bf16 beside a bf16 x).
extern "C" int dewb_moe_router(const void* x, const void* w, const float* bias, const float* logit_bias, const int* positions, int T, int d, int E,
                               int k, int groups, int keep, int best, float fill, int score, int norm, float scaling, float* weights, int* ids, int* rank, int* counts, int x_fp32,
                               int w_fp32, void* stream_ptr) {
  if (T <= 0) return 0;
  const Choice c{bias, logit_bias, E, k, groups, keep, best, fill, score, norm, scaling, weights, ids, rank, counts};
  if (!choice_ok(c) || d < 1 || (x_fp32 && !w_fp32)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bool vec = d % 4 == 0 && aligned(x, 16) && aligned(w, 16);
  const float* wf = static_cast<const float*>(w);
  const bf16 *xb = static_cast<const bf16*>(x), *wb = static_cast<const bf16*>(w);
  if (x_fp32) {
    const float* xf = static_cast<const float*>(x);
    return vec ? router<float, float, 4>(xf, wf, positions, T, d, c, stream) : router<float, float, 1>(xf, wf, positions, T, d, c, stream);
  }
  if (w_fp32) return vec ? router<bf16, float, 4>(xb, wf, positions, T, d, c, stream) : router<bf16, float, 1>(xb, wf, positions, T, d, c, stream);
  if (vec && d % 8 == 0) return router<bf16, bf16, 8>(xb, wb, positions, T, d, c, stream);
  return vec ? router<bf16, bf16, 4>(xb, wb, positions, T, d, c, stream) : router<bf16, bf16, 1>(xb, wb, positions, T, d, c, stream);
}

// x [T, d] -> rows [tiles * 128, d] sorted by expert, place [T, k], tile_group [tiles], offsets [E + 1]; gate [T] with gate_w [d] (both or neither).
extern "C" int dewb_moe_gather(const void* x, const int* ids, const int* rank, const int* counts, const void* gate_w, void* rows_out, int* place,
                               int* tile_group, int* offsets, float* gate, int T, int d, int E, int k, int tiles, int fp32, void* stream_ptr) {
  if (T <= 0) return 0;
  if (d < 1 || E < 1 || E > MAX_E || k < 1 || k > MAX_K || tiles < 1 || tiles > (1 << 23) || (gate_w == nullptr) != (gate == nullptr)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (fp32) return gather<float>(x, ids, rank, counts, gate_w, rows_out, place, tile_group, offsets, gate, T, d, E, k, tiles, stream);
  return gather<bf16>(x, ids, rank, counts, gate_w, rows_out, place, tile_group, offsets, gate, T, d, E, k, tiles, stream);
}

extern "C" int dewb_moe_gemm(const void* a, const void* w, void* out, const int* tile_group, const int* offsets, const int* counts, int tiles, int N,
                             int K, int fp32, void* stream_ptr) {
  if (tiles <= 0 || N <= 0 || K <= 0) return 0;
  if (tiles > 32767) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const dim3 grid((N + 63) / 64, tiles * (BLOCK / 64));
  if (fp32) moe_gemm_kernel<float><<<grid, THREADS, 0, stream>>>(static_cast<const float*>(a), static_cast<const float*>(w), static_cast<float*>(out),
                                                                 tile_group, offsets, counts, N, K);
  else moe_gemm_kernel<bf16><<<grid, THREADS, 0, stream>>>(static_cast<const bf16*>(a), static_cast<const bf16*>(w), static_cast<bf16*>(out), tile_group,
                                                           offsets, counts, N, K);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dewb_moe_glu(const void* gu, void* out, const int* tile_group, const int* offsets, const int* counts, int tiles, int F, int fp32,
                            void* stream_ptr) {
  if (tiles <= 0 || F <= 0) return 0;
  if (tiles > (1 << 23)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bool a16 = aligned(gu, 16) && aligned(out, 16);
  const int blocks = tiles * (BLOCK / WARPS);
#define DEWB_MGLU(TT, VV) moe_glu_kernel<TT, VV><<<blocks, THREADS, 0, stream>>>(static_cast<const TT*>(gu), static_cast<TT*>(out), tile_group, offsets, counts, F)
  if (fp32) { if (a16 && F % 4 == 0) DEWB_MGLU(float, 4); else DEWB_MGLU(float, 1); }
  else { if (a16 && F % 8 == 0) DEWB_MGLU(bf16, 8); else if (a16 && F % 4 == 0) DEWB_MGLU(bf16, 4); else DEWB_MGLU(bf16, 1); }
#undef DEWB_MGLU
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dewb_moe_combine(const void* y, const float* weights, const int* place, const void* shared, const float* gate, void* out, int T, int d,
                                int k, int fp32, void* stream_ptr) {
  if (T <= 0) return 0;
  if (d < 1 || k < 1 || k > MAX_K) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bool a16 = aligned(y, 16) && aligned(shared, 16) && aligned(out, 16);
  const int v = a16 && !fp32 && d % 8 == 0 ? 8 : a16 && d % 4 == 0 ? 4 : 1;
  const int blocks = (d + COMBINE * v - 1) / (COMBINE * v);
  if (blocks > 65535) return -3;
  const dim3 grid(T, blocks);
#define DEWB_COMB(TT, VV) moe_combine_kernel<TT, VV><<<grid, COMBINE, 0, stream>>>(static_cast<const TT*>(y), weights, place, static_cast<const TT*>(shared), \
    gate, static_cast<TT*>(out), d, k)
  if (fp32) { if (v == 4) DEWB_COMB(float, 4); else DEWB_COMB(float, 1); }
  else { if (v == 8) DEWB_COMB(bf16, 8); else if (v == 4) DEWB_COMB(bf16, 4); else DEWB_COMB(bf16, 1); }
#undef DEWB_COMB
  return static_cast<int>(cudaGetLastError());
}
