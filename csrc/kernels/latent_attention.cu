// Latent attention in generation, for sm_100a: a token leaves one row [latent | rotated key part] for all heads, in pages W values wide: rank + rot
// padded with zeros to a multiple of 16, and 8 more, so that rows copied to shared memory as they lie start on different banks.
//
//   latent_rows      from the input projection [tokens, query latent | latent | key part | ...]: RMS norm of the query latent and of the latent, the
//                    rotation of the key part (by the call's table of cosines and sines), and the append of the row to its page
//   rotate_tail      the last columns of every query head rotated in place (prompts: the heads meet their keys in full width)
//   head_product     one product per head, out[t, h, :] = a[t, h, :] w[h]: queries into the latents' space (with the rotated tail of each head beside
//                    them) and latents out of it, times the sigmoid of a gate.  bf16 on the tensor cores (mma.sync: a decode step has too few rows for
//                    tcgen05), fp32 and ragged sizes on the CUDA cores
//   latent_attend    causal attention of a call's tokens against the rows' latents (decode steps, mixed positions): 16 or 32 rows of work (token,
//                    head) a CTA, tiles of 32 latents through a ring of bulk copies, each read once for scores and values, keys split over CTAs
//   latent_combine   merges the splits
//   latent_gather    pages -> dense latents and key parts of every row (a prompt's later portions, whose keys are formed in full width)
//
// Positions below 0 are padding: nothing is appended for them and their outputs are zero.  Norms, angles, scores and sums are fp32.  Compiled without
// fast math.
#include <climits>
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/mma_bf16.cuh"
#include "../common/ptx.cuh"
#include "../common/rows.cuh"

namespace dewb {
namespace latent {

using namespace rows;
using namespace mma16;

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }

struct Pool {
  const int* table;       // [store rows, max_pages]
  int page_size, max_pages;
  const int* row_ids;     // store row of each call row, null: the same
};

__device__ __forceinline__ long long pool_token(const Pool& p, int row, int pos) {
  const int r = p.row_ids == nullptr ? row : p.row_ids[row];
  return static_cast<long long>(p.table[static_cast<long long>(r) * p.max_pages + pos / p.page_size]) * p.page_size + pos % p.page_size;
}

// Column j of a head's rotated part (`x` its first column): pairs are neighbours, or the two halves.
template <typename T>
__device__ __forceinline__ float turned(const T* x, int j, const float2* angle, int dims, int interleaved) {
  if (j >= dims) return ld(x + j);
  const int half = dims / 2;
  const bool low = interleaved ? j % 2 == 0 : j < half;
  const float2 t = angle[interleaved ? j / 2 : low ? j : j - half];
  const float mine = ld(x + j), other = ld(x + (interleaved ? (low ? j + 1 : j - 1) : low ? j + half : j - half));
  return low ? mine * t.x - other * t.y : mine * t.x + other * t.y;
}

constexpr int ROW_THREADS = 128;

// One block a token.  z [tokens, stride]; cq [tokens, q_rank]; c [tokens, rank]; kr [tokens, rot]; pool [*, W].
template <typename T, int V>
__global__ void __launch_bounds__(ROW_THREADS)
latent_rows_kernel(const T* __restrict__ z, long long stride, const T* __restrict__ qw, const T* __restrict__ cw, float eps,
                   const float2* __restrict__ table, int dims, int interleaved, const int* __restrict__ positions, int S, int q_rank, int rank, int rot,
                   int W, T* __restrict__ cq, T* __restrict__ c, T* __restrict__ kr, T* __restrict__ pool, Pool pages) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int pos = positions[t];
  const T* src = z + t * stride;
  auto norm = [&](const T* x, const T* w, int n, T* dst, T* dst2) {
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < n; i += ROW_THREADS * V) {
      float a[V];
      load_v<V>(x + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += a[j] * a[j];
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / n + eps);
    for (int i = threadIdx.x * V; i < n; i += ROW_THREADS * V) {
      float a[V], b[V];
      load_v<V>(x + i, a);
      load_v<V>(w + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] = a[j] * r * b[j];
      store_v<V>(dst + i, a);
      if (dst2 != nullptr) store_v<V>(dst2 + i, a);
    }
  };
  if (q_rank > 0) norm(src, qw, q_rank, cq + t * q_rank, nullptr);
  T* row = pos >= 0 ? pool + pool_token(pages, static_cast<int>(t / S), pos) * W : nullptr;
  norm(src + q_rank, cw, rank, c + t * rank, row);
  const T* part = src + q_rank + rank;
  const float2* angle = table + t * (dims / 2);
  for (int j = threadIdx.x; j < W - rank; j += ROW_THREADS) {
    const float v = j < rot ? turned(part, j, angle, dims, interleaved) : 0.f;
    if (j < rot) st(kr + t * rot + j, v);
    if (row != nullptr) st(row + rank + j, v);
  }
}

// x [tokens, H, width]: columns [first, first + dims) of every head turned in place; a thread a pair
template <typename T>
__global__ void __launch_bounds__(256)
rotate_tail_kernel(T* __restrict__ x, const float2* __restrict__ table, long long pairs, int H, int width, int first, int half, int interleaved) {
  const long long at = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (at >= pairs) return;
  const int i = static_cast<int>(at % half);
  const long long head = at / half;                  // token * H + head
  const float2 t = table[head / H * half + i];
  T* u = x + head * width + first + (interleaved ? 2 * i : i);
  T* v = u + (interleaved ? 1 : half);
  const float a = ld(u), b = ld(v);
  st(u, a * t.x - b * t.y);
  st(v, b * t.x + a * t.y);
}

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// One product per head.  a [T, H, *], w [H, N, K] (rows w_ld apart) or, TRANS, [H, K, N]; out [T, H, *]; strides in elements.
template <typename T>
struct HeadProduct {
  const T* a;
  long long a_token, a_head;
  const T* w;
  long long w_head, w_ld;
  const T* gate;                   // [T, *] or null: out times sigmoid(gate[t, h * N + n])
  long long gate_token;
  T* out;
  long long out_token, out_head;
  int tokens, H, N, K;
  const float2* table;             // not null: columns [N, N + pad) of out are the rotated columns [K, K + rot) of a, then zeros
  int rot, pad, dims, interleaved;
  int pairs;                       // columns of out and gate can be moved in pairs
};

// Part `part` of the tail: TAIL columns of up to 64 rows
constexpr int TAIL = 16;

template <typename T>
__device__ __forceinline__ void tail_columns(const HeadProduct<T>& p, int t0, int part, int h, int threads) {
  const int c0 = part * TAIL, n = min(TAIL, p.pad - c0), end = min(64, p.tokens - t0) * n;
#pragma unroll 4
  for (int i = threadIdx.x; i < end; i += threads) {
    const int r = i / n, j = c0 + i - r * n;
    const long long t = t0 + r;
    const float v = j < p.rot ? turned(p.a + t * p.a_token + h * p.a_head + p.K, j, p.table + t * (p.dims / 2), p.dims, p.interleaved) : 0.f;
    st(p.out + t * p.out_token + h * p.out_head + p.N + j, v);
  }
}

// grid (ceil(N / 64) (+ ceil(pad / TAIL) with a table), ceil(tokens / 64), H)
template <typename T, bool TRANS>
__global__ void __launch_bounds__(256)
head_product_kernel(HeadProduct<T> p) {
  constexpr int M = 64, NT = 64, KT = 16;
  __shared__ __align__(16) float sa[KT][M + 4], sw[KT][NT + 4];
  const int t0 = blockIdx.y * M, n0 = blockIdx.x * NT, h = blockIdx.z;
  if (n0 >= p.N) { tail_columns(p, t0, blockIdx.x - (p.N + NT - 1) / NT, h, 256); return; }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += KT) {
    for (int i = threadIdx.x; i < M * KT; i += 256) {
      const int r = i / KT, c = i - r * KT;
      sa[c][r] = t0 + r < p.tokens && k0 + c < p.K ? ld(p.a + (t0 + r) * p.a_token + h * p.a_head + k0 + c) : 0.f;
    }
    for (int i = threadIdx.x; i < NT * KT; i += 256) {
      const int n = TRANS ? i % NT : i / KT, c = TRANS ? i / NT : i - n * KT;
      sw[c][n] = n0 + n < p.N && k0 + c < p.K ? ld(p.w + h * p.w_head + (TRANS ? (k0 + c) * p.w_ld + n0 + n : (n0 + n) * p.w_ld + k0 + c)) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < KT; ++c) {
      const float4 x4 = *reinterpret_cast<const float4*>(&sa[c][ty * 4]), y4 = *reinterpret_cast<const float4*>(&sw[c][tx * 4]);
      const float x[4] = {x4.x, x4.y, x4.z, x4.w}, y[4] = {y4.x, y4.y, y4.z, y4.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += x[i] * y[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const long long t = t0 + ty * 4 + i;
    if (t >= p.tokens) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      float v = acc[i][j];
      if (p.gate != nullptr) v *= sigmoid(ld(p.gate + t * p.gate_token + static_cast<long long>(h) * p.N + n));
      st(p.out + t * p.out_token + h * p.out_head + n, v);
    }
  }
}

__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool live) {
  const int n = live ? 16 : 0;                     // 0: the 16 bytes are filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// The same on the tensor cores: 64 x 64 tiles, 8 warps of 16 rows and 32 columns, K in pieces of 128 through a ring.  Every 16-byte piece of the operands
// is aligned and whole (K, and N for TRANS, multiples of 8).
constexpr int PK = 128, PST = PK + 8, WST = 72;    // smem row strides: pieces of a and w, and of a TRANS w (its rows are columns of the product)
constexpr int P_STAGES = 3, P_THREADS = 256, P_STAGE = 64 * PST + (64 * PST > PK * WST ? 64 * PST : PK * WST);

template <bool TRANS>
__global__ void __launch_bounds__(P_THREADS)
head_product_mma_kernel(HeadProduct<bf16> p) {
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* ring = reinterpret_cast<bf16*>(raw);
  const int t0 = blockIdx.y * 64, n0 = blockIdx.x * 64, h = blockIdx.z;
  if (n0 >= p.N) { tail_columns(p, t0, blockIdx.x - (p.N + 63) / 64, h, P_THREADS); return; }
  const int tid = threadIdx.x, lane = tid & 31, warp = (tid >> 5) & 3, half = tid >> 7;
  const int steps = (p.K + PK - 1) / PK;
  auto fetch = [&](int s) {
    if (s < steps) {
      bf16* sa = ring + (s % P_STAGES) * P_STAGE;
      bf16* sw = sa + 64 * PST;
      const int k0 = s * PK;
#pragma unroll
      for (int i = 0; i < 64 * PK / 8 / P_THREADS; ++i) {
        const int at = i * P_THREADS + tid, r = at / (PK / 8), c = at % (PK / 8) * 8;
        const bool la = t0 + r < p.tokens && k0 + c < p.K;
        cp16(smem_addr(sa + r * PST + c), la ? p.a + (t0 + r) * p.a_token + h * p.a_head + k0 + c : p.a, la);
        const int wr = TRANS ? at >> 3 : r, wc = TRANS ? (at & 7) * 8 : c;
        const bool lw = TRANS ? k0 + wr < p.K && n0 + wc < p.N : n0 + wr < p.N && k0 + wc < p.K;
        cp16(smem_addr(sw + wr * (TRANS ? WST : PST) + wc),
             lw ? p.w + h * p.w_head + (TRANS ? (k0 + wr) * p.w_ld + n0 + wc : (n0 + wr) * p.w_ld + k0 + wc) : p.w, lw);
      }
    }
    cp_commit();
  };
  float acc[4][4] = {};
#pragma unroll
  for (int s = 0; s < P_STAGES - 1; ++s) fetch(s);
  for (int s = 0; s < steps; ++s) {
    cp_wait<P_STAGES - 2>();
    __syncthreads();
    fetch(s + P_STAGES - 1);
    const bf16* sa = ring + (s % P_STAGES) * P_STAGE;
    const bf16* sw = sa + 64 * PST;
#pragma unroll
    for (int kk = 0; kk < PK; kk += 16) {
      uint32_t a[4], b[2][4];
      ldsm4(a, smem_addr(sa + (warp * 16 + (lane & 15)) * PST + kk + (lane >> 4) * 8));
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int n = half * 32 + j * 16;
        if (TRANS) ldsm4_t(b[j], smem_addr(sw + (kk + (lane & 15)) * WST + n + (lane >> 4) * 8));
        else ldsm4(b[j], smem_addr(sw + (n + (lane & 7) + (lane >> 4) * 8) * PST + kk + ((lane >> 3) & 1) * 8));
      }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma(acc[2 * j], a, b[j][0], b[j][1]);
        mma(acc[2 * j + 1], a, b[j][2], b[j][3]);
      }
    }
  }
  cp_wait<0>();
  const int lg = lane >> 2, t2 = (lane & 3) * 2;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const long long t = t0 + warp * 16 + lg + 8 * e;
    if (t >= p.tokens) continue;
    if (p.pairs) {                                     // pairs of columns; every gate is under way before the first is used
      uint32_t z[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + half * 32 + j * 8 + t2;
        z[j] = p.gate != nullptr && n < p.N ? *reinterpret_cast<const uint32_t*>(p.gate + t * p.gate_token + static_cast<long long>(h) * p.N + n) : 0u;
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + half * 32 + j * 8 + t2;
        float a = acc[j][2 * e], b = acc[j][2 * e + 1];
        if (p.gate != nullptr) { a *= sigmoid(lo_f(z[j])); b *= sigmoid(hi_f(z[j])); }
        if (n < p.N) *reinterpret_cast<uint32_t*>(p.out + t * p.out_token + h * p.out_head + n) = pack2(a, b);
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int n = n0 + half * 32 + j * 8 + t2 + q;
        if (n >= p.N) continue;
        float v = acc[j][2 * e + q];
        if (p.gate != nullptr) v *= sigmoid(ld(p.gate + t * p.gate_token + static_cast<long long>(h) * p.N + n));
        st(p.out + t * p.out_token + h * p.out_head + n, v);
      }
  }
}

// ---- attention against the latents: 17 warps.  Warp 16 brings tiles of 32 rows into a ring, one bulk copy a tile (a row, where pages do not hold whole
// tiles).  Warps 0..7 form scores: a warp takes a quarter of the W columns and half of the tile's keys, and leaves its part in shared memory.  Warps 8..15
// add the parts up, keep the online softmax and the sums (NV * 8 latent columns each), and free the stage.  Scores of one tile and softmax and values of
// the one before run at the same time.  KS: 16-column steps of a quarter; MT: tiles of 16 rows of work (token, head).
constexpr int TK = 32, GROUP = 256, A_THREADS = 2 * GROUP + 32, SST = TK + 8, PPT = TK + 8;
constexpr uint32_t FULL = 0xffffffffu;

struct Attend {
  const bf16* q;                   // [R * S, H, W]
  const bf16* pool;                // [*, W]
  const int* positions;            // [R * S]
  bf16* out;                       // [R * S, H, rank] (one split)
  float *part_m, *part_l, *part_acc;      // [R * S * H, splits] (log2 domain) and [..., rank]
  int S, H, W, rank, splits;
  float scale_log2;
  int* err;
};

template <int MT>
constexpr int attend_stages() { return MT == 1 ? 5 : 4; }

template <int STAGES>
struct AttendBars {
  uint64_t k_full[STAGES], k_empty[STAGES], s_full[2], s_empty[2];
  int abort_flag, poisoned;
};

template <int KS, int NV, int MT>
__global__ void __launch_bounds__(A_THREADS, 1)
latent_attend_kernel(Attend p, Pool pages) {
  constexpr int STAGES = attend_stages<MT>(), M = 16 * MT, TPR = GROUP / M, KPT = TK / TPR;
  extern __shared__ __align__(16) uint8_t raw[];
  const int ST = p.W;
  bf16* sk = reinterpret_cast<bf16*>(raw);                       // [STAGES][TK][W]
  float* ss = reinterpret_cast<float*>(sk + STAGES * TK * ST);   // [2][4][M][SST]
  bf16* sp = reinterpret_cast<bf16*>(ss + 2 * 4 * M * SST);      // [2][M][PPT]
  __shared__ AttendBars<STAGES> bars;
  __shared__ float s_alpha[2][M], s_l[M], s_m[M];
  __shared__ int s_pos[M];
  const int row = blockIdx.y, split = blockIdx.z, w0 = blockIdx.x * M, work = p.S * p.H;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) {
    bars.poisoned = *reinterpret_cast<volatile int*>(p.err);
    bars.abort_flag = 0;
    for (int i = 0; i < STAGES; ++i) { mbar_init(&bars.k_full[i], 1); mbar_init(&bars.k_empty[i], 8); }
    for (int i = 0; i < 2; ++i) { mbar_init(&bars.s_full[i], 8); mbar_init(&bars.s_empty[i], 8); }
    fence_barrier_init();
    fence_proxy_async();
  }
  if (tid < M) s_pos[tid] = w0 + tid < work ? p.positions[static_cast<long long>(row) * p.S + (w0 + tid) / p.H] : -1;
  __syncthreads();
  if (bars.poisoned != 0) return;
  volatile int* abort_flag = &bars.abort_flag;
  int last = -1;
  for (int i = 0; i < M; ++i) last = max(last, s_pos[i]);
  const int all = (last + TK) / TK, per = (all + p.splits - 1) / p.splits;
  const int begin = min(all, split * per), tiles = min(all, begin + per) - begin;
  const int lg = lane >> 2, t2 = (lane & 3) * 2;
  if (warp == 16) {
    // ------------------------------------------------------------------ producer
    // Tokens past the last one (a tile whole in a page brings them along, else the last is repeated) meet weights of zero.
    const bool whole = pages.page_size % TK == 0;
    auto source = [&](int t) { return pool_token(pages, row, whole ? (begin + t) * TK : min((begin + t) * TK + lane, last)); };
    long long tok = tiles > 0 ? source(0) : 0;
    int t = 0;
    for (; t < tiles; ++t) {
      const int st = t % STAGES;
      if (!mbar_wait_warp(&bars.k_empty[st], ((t / STAGES) & 1) ^ 1, abort_flag)) { if (lane == 0) atomicCAS(p.err, 0, ERR_WAIT_EMPTY); break; }
      if (lane == 0) mbar_expect_tx(&bars.k_full[st], TK * p.W * 2);
      __syncwarp();
      if (!whole) bulk_load_1d(sk + (st * TK + lane) * ST, p.pool + tok * p.W, p.W * 2, &bars.k_full[st]);
      else if (lane == 0) bulk_load_1d(sk + st * TK * ST, p.pool + tok * p.W, TK * p.W * 2, &bars.k_full[st]);
      if (t + 1 < tiles) tok = source(t + 1);          // the page's number is under way while the ring is full
    }
    if (t < tiles)                                     // gave up: the copies under way still land in this block's memory
      for (int i = max(0, t - STAGES); i < t; ++i) mbar_wait_warp(&bars.k_full[i % STAGES], (i / STAGES) & 1, nullptr);
  } else if (warp < 8) {
    // ------------------------------------------------------------------ scores
    const int kq = warp & 3, kg = warp >> 2, steps = (p.W - 8) / 16, quarter = (steps + 3) / 4, first = kq * quarter, count = max(0, min(quarter, steps - first));
    uint32_t qa[MT][KS][4];                            // this warp's columns of the queries, as A operands
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int w = w0 + m * 16 + lg + 8 * e;
        const bool live = w < work && s_pos[m * 16 + lg + 8 * e] >= 0;
        const bf16* src = p.q + (static_cast<long long>(row) * work + w) * p.W;
#pragma unroll
        for (int k = 0; k < KS; ++k) {
          qa[m][k][e] = live && k < count ? *reinterpret_cast<const uint32_t*>(src + (first + k) * 16 + t2) : 0u;
          qa[m][k][2 + e] = live && k < count ? *reinterpret_cast<const uint32_t*>(src + (first + k) * 16 + 8 + t2) : 0u;
        }
      }
    const uint32_t kaddr = smem_addr(sk) + ((kg * 16 + (lane & 7) + (lane >> 4) * 8) * ST + first * 16 + ((lane >> 3) & 1) * 8) * 2;
    for (int t = 0; t < tiles; ++t) {
      const int st = t % STAGES, b = t & 1;
      if (!mbar_wait_warp(&bars.k_full[st], (t / STAGES) & 1, abort_flag)) { if (lane == 0) atomicCAS(p.err, 0, ERR_WAIT_FULL); break; }
      float* part = ss + b * 4 * M * SST;
      {
        float s[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n) { s[m][n][0] = s[m][n][1] = s[m][n][2] = s[m][n][3] = 0.f; }
        const uint32_t at = kaddr + st * TK * ST * 2;
#pragma unroll
        for (int k = 0; k < KS; ++k)
          if (k < count) {
            uint32_t f[4];
            ldsm4(f, at + k * 32);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma(s[m][0], qa[m][k], f[0], f[1]);
              mma(s[m][1], qa[m][k], f[2], f[3]);
            }
          }
        if (!mbar_wait_warp(&bars.s_empty[b], ((t >> 1) & 1) ^ 1, abort_flag)) { if (lane == 0) atomicCAS(p.err, 0, ERR_WAIT_OTHER); break; }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            float* d = part + (kq * M + m * 16 + lg) * SST + kg * 16 + n * 8 + t2;
            *reinterpret_cast<float2*>(d) = make_float2(s[m][n][0], s[m][n][1]);
            *reinterpret_cast<float2*>(d + 8 * SST) = make_float2(s[m][n][2], s[m][n][3]);
          }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars.s_full[b]);
    }
  }
  float o[MT][NV][4];
  const int v0 = (warp - 8) * NV * 8;
  if (warp >= 8 && warp < 16) {
    // ------------------------------------------------------------------ softmax and sums of latents
    const int bid = tid - GROUP, srow = bid / TPR, skey = (bid % TPR) * KPT, my_pos = s_pos[srow];      // this thread's scores
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < NV; ++n) { o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f; }
    const uint32_t vaddr = smem_addr(sk) + ((lane & 15) * ST + v0 + (lane >> 4) * 8) * 2;
    const uint32_t paddr = smem_addr(sp) + ((lane & 15) * PPT + (lane >> 4) * 8) * 2;
    for (int t = 0; t < tiles; ++t) {
      const int st = t % STAGES, b = t & 1;
      const float* part = ss + b * 4 * M * SST;
      if (ok && !mbar_wait_warp(&bars.s_full[b], (t >> 1) & 1, abort_flag)) { if (lane == 0) atomicCAS(p.err, 0, ERR_WAIT_OTHER); ok = false; }
      if (ok) {
        float v[KPT], mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < KPT; ++i) v[i] = 0.f;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float x[KPT];
          const float* src = part + (q * M + srow) * SST + skey;
          if constexpr (KPT == 4) load_v<4>(src, x);
          else { const float2 y = *reinterpret_cast<const float2*>(src); x[0] = y.x; x[1] = y.y; }
#pragma unroll
          for (int i = 0; i < KPT; ++i) v[i] += x[i];
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(&bars.s_empty[b]);
#pragma unroll
        for (int i = 0; i < KPT; ++i) {
          v[i] = (begin + t) * TK + skey + i <= my_pos ? v[i] * p.scale_log2 : -INFINITY;
          mx = fmaxf(mx, v[i]);
        }
#pragma unroll
        for (int d = TPR / 2; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(FULL, mx, d));
        const float mn = fmaxf(m_run, mx), base = mn == -INFINITY ? 0.f : mn, alpha = exp2f(m_run - base);
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < KPT; ++i) { v[i] = exp2f(v[i] - base); sum += v[i]; }
        l_run = l_run * alpha + sum;                     // (this thread's keys alone: the parts meet at the end)
        m_run = mn;
#pragma unroll
        for (int i = 0; i < KPT; i += 2) *reinterpret_cast<uint32_t*>(sp + (b * M + srow) * PPT + skey + i) = pack2(v[i], v[i + 1]);
        if (bid % TPR == 0) s_alpha[b][srow] = alpha;
      }
      // the eight warps meet once a tile: the two buffers of weights take turns
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (ok && !mbar_wait_warp(&bars.k_full[st], (t / STAGES) & 1, abort_flag)) { if (lane == 0) atomicCAS(p.err, 0, ERR_WAIT_FULL); ok = false; }
      if (!ok) continue;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float a0 = s_alpha[b][m * 16 + lg], a1 = s_alpha[b][m * 16 + lg + 8];
        if (__any_sync(FULL, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
          for (int n = 0; n < NV; ++n) { o[m][n][0] *= a0; o[m][n][1] *= a0; o[m][n][2] *= a1; o[m][n][3] *= a1; }
        }
      }
#pragma unroll
      for (int kk = 0; kk < TK; kk += 16) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm4(a[m], paddr + ((b * M + m * 16) * PPT + kk) * 2);
#pragma unroll
        for (int n = 0; n < NV; n += 2)
          if (v0 + n * 8 < p.rank) {
            uint32_t f[4];
            ldsm4_t(f, vaddr + ((st * TK + kk) * ST + n * 8) * 2);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma(o[m][n], a[m], f[0], f[1]);
              mma(o[m][n + 1], a[m], f[2], f[3]);
            }
          }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars.k_empty[st]);
    }
#pragma unroll
    for (int d = TPR / 2; d > 0; d >>= 1) l_run += __shfl_xor_sync(FULL, l_run, d);
    if (bid % TPR == 0) { s_l[srow] = l_run; s_m[srow] = m_run; }
  }
  __syncthreads();
  if (warp < 8 || warp >= 16) {
    if (p.splits > 1 && tid < M && w0 + tid < work) {
      const long long at = (static_cast<long long>(row) * work + w0 + tid) * p.splits + split;
      p.part_m[at] = s_m[tid];
      p.part_l[at] = s_l[tid];
    }
    return;
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = m * 16 + lg + 8 * e;
      if (w0 + r >= work) continue;
      const long long at = static_cast<long long>(row) * work + w0 + r;
      const float l = s_l[r], inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
      for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int c = v0 + n * 8 + t2 + q;
          if (c >= p.rank) continue;
          if (p.splits == 1) p.out[at * p.rank + c] = __float2bfloat16(o[m][n][2 * e + q] * inv);
          else p.part_acc[(at * p.splits + split) * p.rank + c] = o[m][n][2 * e + q];
        }
    }
}

// a block a (token, head)
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_m, const float* __restrict__ part_l, const float* __restrict__ part_acc, bf16* __restrict__ out,
                      int splits, int rank) {
  const long long at = blockIdx.x;
  float top = -INFINITY, l = 0.f;
  for (int s = 0; s < splits; ++s) top = fmaxf(top, part_m[at * splits + s]);
  for (int s = 0; s < splits; ++s) {
    const float m = part_m[at * splits + s];
    if (m > -INFINITY) l += part_l[at * splits + s] * exp2f(m - top);
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int c = threadIdx.x; c < rank; c += 128) {
    float a = 0.f;
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
      const float m = part_m[at * splits + s];
      if (m > -INFINITY) a += part_acc[(at * splits + s) * rank + c] * exp2f(m - top);
    }
    out[at * rank + c] = __float2bfloat16(a * inv);
  }
}

// grid (ceil(T / 8), R), a warp a token: c [R, T, rank], kr [R, T, rot]; tokens past a row's length read as zeros
template <typename T, int V>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const T* __restrict__ pool, const int* __restrict__ lengths, Pool pages, int total, int rank, int rot, int W, T* __restrict__ c,
                     T* __restrict__ kr) {
  const int pos = blockIdx.x * 8 + (threadIdx.x >> 5), row = blockIdx.y, lane = threadIdx.x & 31;
  if (pos >= total) return;
  const long long at = static_cast<long long>(row) * total + pos;
  const T* src = pos < lengths[row] ? pool + pool_token(pages, row, pos) * W : nullptr;
  for (int i = lane * V; i < rank + rot; i += 32 * V) {
    float a[V];
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = 0.f;
    if (src != nullptr) load_v<V>(src + i, a);
    store_v<V>(i < rank ? c + at * rank + i : kr + at * rot + i - rank, a);
  }
}

template <typename T>
int rows_of(const void* z, long long stride, const void* qw, const void* cw, float eps, const float* table, int dims, int interleaved,
            const int* positions, int R, int S, int q_rank, int rank, int rot, int W, void* cq, void* c, void* kr, void* pool, const Pool& pages,
            cudaStream_t stream) {
  const bool vec = q_rank % 4 == 0 && rank % 4 == 0 && stride % 4 == 0 && W % 4 == 0 && aligned(z, 16) && aligned(qw, 16) && aligned(cw, 16) &&
                   aligned(cq, 16) && aligned(c, 16) && aligned(pool, 16);
  const bool vec8 = vec && sizeof(T) == 2 && q_rank % 8 == 0 && rank % 8 == 0 && stride % 8 == 0 && W % 8 == 0;
#define DEWB_ROWS(VV) latent_rows_kernel<T, VV><<<static_cast<unsigned>(R) * static_cast<unsigned>(S), ROW_THREADS, 0, stream>>>(static_cast<const T*>(z), \
    stride, static_cast<const T*>(qw), static_cast<const T*>(cw), eps, reinterpret_cast<const float2*>(table), dims, interleaved, positions, S, q_rank, rank, \
    rot, W, static_cast<T*>(cq), static_cast<T*>(c), static_cast<T*>(kr), static_cast<T*>(pool), pages)
  if constexpr (sizeof(T) == 2) { if (vec8) DEWB_ROWS(8); else if (vec) DEWB_ROWS(4); else DEWB_ROWS(1); }
  else { if (vec) DEWB_ROWS(4); else DEWB_ROWS(1); }
#undef DEWB_ROWS
  return static_cast<int>(cudaGetLastError());
}

template <int KS, int NV, int MT>
int attend(const Attend& p, const Pool& pages, int R, cudaStream_t stream) {
  constexpr int M = 16 * MT;
  const int smem = attend_stages<MT>() * TK * p.W * 2 + 2 * 4 * M * SST * 4 + 2 * M * PPT * 2;
  cudaError_t e = cudaFuncSetAttribute(latent_attend_kernel<KS, NV, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  const long long blocks = (static_cast<long long>(p.S) * p.H + M - 1) / M;
  latent_attend_kernel<KS, NV, MT><<<dim3(static_cast<unsigned>(blocks), R, p.splits), A_THREADS, smem, stream>>>(p, pages);
  e = cudaGetLastError();
  if (e != cudaSuccess || p.splits == 1) return static_cast<int>(e);
  latent_combine_kernel<<<static_cast<unsigned>(R) * static_cast<unsigned>(p.S) * p.H, 128, 0, stream>>>(p.part_m, p.part_l, p.part_acc, p.out, p.splits, p.rank);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int product(HeadProduct<T> p, int trans, cudaStream_t stream) {
  p.pairs = p.N % 2 == 0 && p.out_token % 2 == 0 && p.out_head % 2 == 0 && p.gate_token % 2 == 0 && aligned(p.out, 4) && aligned(p.gate, 4);
  const dim3 grid((p.N + 63) / 64 + (p.table != nullptr ? (p.pad + TAIL - 1) / TAIL : 0), (p.tokens + 63) / 64, p.H);
  if constexpr (sizeof(T) == 2) {
    const bool whole = p.K % 8 == 0 && (!trans || p.N % 8 == 0) && p.a_token % 8 == 0 && p.a_head % 8 == 0 && p.w_head % 8 == 0 && p.w_ld % 8 == 0 &&
                       aligned(p.a, 16) && aligned(p.w, 16);
    if (whole) {
      const int smem = P_STAGES * P_STAGE * 2;
      cudaError_t e = trans ? cudaFuncSetAttribute(head_product_mma_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem)
                            : cudaFuncSetAttribute(head_product_mma_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return static_cast<int>(e);
      if (trans) head_product_mma_kernel<true><<<grid, P_THREADS, smem, stream>>>(p);
      else head_product_mma_kernel<false><<<grid, P_THREADS, smem, stream>>>(p);
      return static_cast<int>(cudaGetLastError());
    }
  }
  if (trans) head_product_kernel<T, true><<<grid, 256, 0, stream>>>(p);
  else head_product_kernel<T, false><<<grid, 256, 0, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace latent
}  // namespace dewb

using namespace dewb::latent;

// z [R * S, stride]: query latent (q_rank, may be 0) | latent (rank) | key part (rot) -> cq [R * S, q_rank], c [R * S, rank], kr [R * S, rot] and the
// pages pool [*, page_size, W].  qw [q_rank], cw [rank]: the norms' weights; table [R * S, dims / 2, 2].
extern "C" int dewb_latent_rows(const void* z, long long stride, const void* qw, const void* cw, float eps, const float* table, int dims,
                                int interleaved, const int* positions, int R, int S, int q_rank, int rank, int rot, int W, void* cq, void* c, void* kr,
                                void* pool, const int* page_table, int page_size, int max_pages, const int* row_ids, int fp32, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (q_rank < 0 || rank < 1 || rot < 2 || dims < 2 || dims % 2 || dims > rot || W < rank + rot || stride < static_cast<long long>(q_rank) + rank + rot || page_size < 1 ||
      max_pages < 1 || table == nullptr)
    return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Pool pages{page_table, page_size, max_pages, row_ids};
  if (fp32) return rows_of<float>(z, stride, qw, cw, eps, table, dims, interleaved, positions, R, S, q_rank, rank, rot, W, cq, c, kr, pool, pages, stream);
  return rows_of<bf16>(z, stride, qw, cw, eps, table, dims, interleaved, positions, R, S, q_rank, rank, rot, W, cq, c, kr, pool, pages, stream);
}

// x [tokens, H, width]: the columns [first, first + dims) of every head turned by table [tokens, dims / 2, 2], in place
extern "C" int dewb_rotate_tail(void* x, const float* table, long long tokens, int H, int width, int first, int dims, int interleaved, int fp32,
                                void* stream_ptr) {
  if (tokens <= 0) return 0;
  if (H < 1 || dims < 2 || dims % 2 || first < 0 || first + dims > width) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const long long pairs = tokens * H * (dims / 2), blocks = (pairs + 255) / 256;
  if (blocks > 0x7fffffffll) return -3;
  const float2* t = reinterpret_cast<const float2*>(table);
  if (fp32) rotate_tail_kernel<float><<<static_cast<unsigned>(blocks), 256, 0, stream>>>(static_cast<float*>(x), t, pairs, H, width, first, dims / 2, interleaved);
  else rotate_tail_kernel<bf16><<<static_cast<unsigned>(blocks), 256, 0, stream>>>(static_cast<bf16*>(x), t, pairs, H, width, first, dims / 2, interleaved);
  return static_cast<int>(cudaGetLastError());
}

// out[t, h, n] = sum_k a[t, h, k] w[h, n, k] (`trans`: w[h, k, n]), times sigmoid(gate[t, h * N + n]) where gate is not null; with a table the
// columns [N, N + pad) of out are the columns [K, K + rot) of a, the first `dims` of them turned, and then zeros.
extern "C" int dewb_head_product(const void* a, long long a_token, long long a_head, const void* w, long long w_head, long long w_ld, int trans,
                                 const void* gate, long long gate_token, void* out, long long out_token, long long out_head, int tokens, int H, int N,
                                 int K, const float* table, int rot, int pad, int dims, int interleaved, int fp32, void* stream_ptr) {
  if (tokens <= 0) return 0;
  if (H < 1 || H > 65535 || N < 1 || K < 1 || tokens > 65535 * 64 || (table != nullptr && (dims < 2 || dims % 2 || rot < dims || pad < rot))) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const float2* t = reinterpret_cast<const float2*>(table);
  if (fp32) return product(HeadProduct<float>{static_cast<const float*>(a), a_token, a_head, static_cast<const float*>(w), w_head, w_ld,
                                              static_cast<const float*>(gate), gate_token, static_cast<float*>(out), out_token, out_head, tokens, H, N, K, t, rot,
                                              pad, dims, interleaved, 0}, trans, stream);
  return product(HeadProduct<dewb::rows::bf16>{static_cast<const dewb::rows::bf16*>(a), a_token, a_head, static_cast<const dewb::rows::bf16*>(w), w_head, w_ld,
                                               static_cast<const dewb::rows::bf16*>(gate), gate_token, static_cast<dewb::rows::bf16*>(out), out_token, out_head,
                                               tokens, H, N, K, t, rot, pad, dims, interleaved, 0}, trans, stream);
}

// q [R * S, H, W] (bf16) against the rows' latents in pool [*, page_size, W] -> out [R * S, H, rank]; W a multiple of 16 plus 8, at most 584, rank at
// most 512.  Scratch for splits > 1 (fp32): part_m, part_l [R * S * H * splits], part_acc [... * rank].  `wide`: 32 rows of work a CTA.
extern "C" int dewb_latent_attend(const void* q, const void* pool, const int* positions, int R, int S, int H, int W, int rank, float scale, int splits,
                                  int wide, float* part_m, float* part_l, float* part_acc, void* out, const int* page_table, int page_size,
                                  int max_pages, const int* row_ids, int* err, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (H < 1 || W < 24 || W % 16 != 8 || W > 584 || rank < 1 || rank > W || rank > 512 || splits < 1 || splits > 65535 || R > 65535 || page_size < 1 || max_pages < 1 ||
      !aligned(q, 16) || !aligned(pool, 16) || (splits > 1 && (part_m == nullptr || part_l == nullptr || part_acc == nullptr)))
    return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Pool pages{page_table, page_size, max_pages, row_ids};
  const Attend p{static_cast<const dewb::rows::bf16*>(q), static_cast<const dewb::rows::bf16*>(pool), positions, static_cast<dewb::rows::bf16*>(out), part_m, part_l,
                 part_acc, S, H, W, rank, splits, scale * 1.4426950408889634f, err};
  if (W <= 200 && rank <= 128) return wide ? attend<3, 2, 2>(p, pages, R, stream) : attend<3, 2, 1>(p, pages, R, stream);
  if (W <= 328 && rank <= 256) return wide ? attend<5, 4, 2>(p, pages, R, stream) : attend<5, 4, 1>(p, pages, R, stream);
  return wide ? attend<9, 8, 2>(p, pages, R, stream) : attend<9, 8, 1>(p, pages, R, stream);
}

// pool [*, page_size, W] -> c [R, total, rank], kr [R, total, rot]: the first `total` tokens of every row, zeros past lengths[row]
extern "C" int dewb_latent_gather(const void* pool, const int* lengths, int R, int total, int rank, int rot, int W, void* c, void* kr,
                                  const int* page_table, int page_size, int max_pages, const int* row_ids, int fp32, void* stream_ptr) {
  if (R <= 0 || total <= 0) return 0;
  if (rank < 1 || rot < 1 || W < rank + rot || page_size < 1 || max_pages < 1 || R > 65535) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Pool pages{page_table, page_size, max_pages, row_ids};
  const dim3 grid((total + 7) / 8, R);
  const bool a16 = aligned(pool, 16) && aligned(c, 16) && aligned(kr, 16);
#define DEWB_LG(TT, VV) latent_gather_kernel<TT, VV><<<grid, 256, 0, stream>>>(static_cast<const TT*>(pool), lengths, pages, total, rank, rot, W, \
    static_cast<TT*>(c), static_cast<TT*>(kr))
  if (fp32) { if (a16 && rank % 4 == 0 && rot % 4 == 0 && W % 4 == 0) DEWB_LG(float, 4); else DEWB_LG(float, 1); }
  else { if (a16 && rank % 8 == 0 && rot % 8 == 0 && W % 8 == 0) DEWB_LG(dewb::rows::bf16, 8); else DEWB_LG(dewb::rows::bf16, 1); }
#undef DEWB_LG
  return static_cast<int>(cudaGetLastError());
}
