// Attention against a paged cache for any head widths, and the projection epilogue in front of it, for sm_100a.
//
//   qk_norm_append   from the packed projection [tokens, H dk + G dk + G dv]: RMS norm of q over all its heads at once and of k likewise
//                    (weights may be null: no norm), the query temperature 1 + coef ln(floor((p + 1) / every) + 1), the copy into heads
//                    of the cache's (padded) width, and the append of keys and values to the page pools
//   head_norm_append   the same for per-head norms (one weight for all heads, or no weight), with the projection's bias added on the way, rows that
//                    carry more columns than the heads (gates), layers that read another layer's keys and values (queries alone), and the rotation
//                    of the first columns of every query and key head by a call's table of cosines and sines
//   rotary_angles    that table, from the positions and the pairs' frequencies
//   head_gate        heads of the cache's width times a sigmoid of one number per head, packed to their own width
//   paged_attend     causal attention of a call's tokens against everything the cache holds of their rows (any start positions; a decode
//                    step is the case of one token per row); scores, softmax and sums in fp32 on the CUDA cores.  It is the fp32 form,
//                    and takes the head widths the tensor-core kernels do not.
//   paged_attend_mma   the same on the tensor cores for bf16 pools 64, 128 or 256 wide (a prompt's later portions, mixed start positions)
//   Both take chunks (a query sees no key from before the start of its chunk of positions), a window beside which the row's first keys may stay
//   visible, a factor per head on the scores, a soft cap on them, a learned sink per head in the denominator, and a gate per head on the output;
//   instead of the softmax, every visible key may weigh the sigmoid of its score plus a number per head, with no sum over the keys.
//
// A query's row of work is (token, head of its group), so a group's heads share the key and value tiles.  Positions below 0 are padding:
// nothing is appended for them and their outputs are zero.  Compiled without fast math.
#include <climits>
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/mma_bf16.cuh"
#include "../common/rows.cuh"

namespace dewb {
namespace paged {

using namespace rows;

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

constexpr int PREP_THREADS = 128;

// grid (tokens, 3): part 0 the queries, 1 the keys, 2 the values.  `packed` [tokens, H + 2 G, D] receives all three; D >= dk, dv.
template <typename T, int V>
__global__ void __launch_bounds__(PREP_THREADS)
qk_norm_append_kernel(const T* __restrict__ qkv, const T* __restrict__ qw, const T* __restrict__ kw, float eps, float coef, int every,
                      const int* __restrict__ positions, int S, int H, int G, int dk, int dv, int D, T* __restrict__ packed,
                      T* __restrict__ kpool, T* __restrict__ vpool, Pool pool) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int part = blockIdx.y;
  const int heads = part == 0 ? H : G, width = part == 2 ? dv : dk, size = heads * width;
  const T* src = qkv + t * (static_cast<long long>(H + G) * dk + G * dv) + (part == 0 ? 0 : part == 1 ? H * dk : (H + G) * dk);
  const T* w = part == 0 ? qw : part == 1 ? kw : nullptr;
  const int pos = positions[t];
  float r = 1.f;
  if (w != nullptr) {
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < size; i += PREP_THREADS * V) {
      float a[V];
      load_v<V>(src + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += a[j] * a[j];
    }
    r = 1.f / sqrtf(block_sum(ss, red) / size + eps);
  }
  float temp = 1.f;
  if (part == 0 && every > 0 && pos >= 0) temp = 1.f + coef * logf(static_cast<float>((pos + 1) / every + 1));
  T* dst = packed + t * static_cast<long long>(H + 2 * G) * D + static_cast<long long>(part == 0 ? 0 : part == 1 ? H : H + G) * D;
  T* to_pool = nullptr;
  if (part != 0 && pos >= 0) {
    const long long tok = pool_token(pool, static_cast<int>(t / S), pos);
    to_pool = (part == 1 ? kpool : vpool) + tok * G * D;
  }
  const int padded = heads * D;                    // the padding of each head is written as zeros
  for (int i = threadIdx.x * V; i < padded; i += PREP_THREADS * V) {
    const int h = i / D, c = i - h * D;
    float a[V];
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = 0.f;
    if (c < width) {
      load_v<V>(src + h * width + c, a);
      if (w != nullptr) {
        float b[V];
        load_v<V>(w + h * width + c, b);
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] = a[j] * r * b[j];
      }
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] *= temp;
    }
    store_v<V>(dst + i, a);
    if (to_pool != nullptr) store_v<V>(to_pool + i, a);
  }
}

// positions [n] -> out [n, half] (cosine, sine) of position * frequency[i]; the angle is formed in double precision
__global__ void __launch_bounds__(256)
rotary_angles_kernel(const int* __restrict__ positions, const double* __restrict__ frequency, float2* __restrict__ out, long long n, int half) {
  const long long at = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (at >= n * half) return;
  const int p = positions[at / half];
  double s, c;
  sincos(static_cast<double>(p > 0 ? p : 0) * frequency[at % half], &s, &c);
  out[at] = make_float2(static_cast<float>(c), static_cast<float>(s));
}

// The rotation of one call: the first `dims` columns of a head turn by `table` [tokens, dims / 2] (cosine, sine); null: none.
struct Turn {
  const float2* table;
  int dims, interleaved;
};

// V consecutive columns of a head starting at `i`, the bias added and each times the head's `gain` and its weight, with the columns below
// `turn.dims` rotated by this token's angles.  src, b, w point at the head's first column; every column that is read lies within the head.
template <typename T, int V>
__device__ __forceinline__ void head_columns(const T* src, const T* b, const T* w, float gain, int i, const float2* angle, int dims, int interleaved,
                                             float (&a)[V]) {
  auto column = [&](int c) {
    float x = ld(src + c);
    if (b != nullptr) x += ld(b + c);
    return w != nullptr ? x * gain * ld(w + c) : x * gain;
  };
  auto columns = [&](int c, float (&x)[V]) {
    load_v<V>(src + c, x);
    if (b != nullptr) {
      float y[V];
      load_v<V>(b + c, y);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] += y[j];
    }
    if (w != nullptr) {
      float y[V];
      load_v<V>(w + c, y);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] = x[j] * gain * y[j];
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] *= gain;
    }
  };
  columns(i, a);
  if (angle == nullptr || i >= dims) return;
  const int half = dims / 2;
  if (!interleaved && half % V == 0) {
    float other[V];
    const bool low = i < half;
    columns(low ? i + half : i - half, other);
    const float2* t = angle + (low ? i : i - half);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = low ? a[j] * t[j].x - other[j] * t[j].y : a[j] * t[j].x + other[j] * t[j].y;
    return;
  }
  if constexpr (V > 1) {
    if (interleaved) {
#pragma unroll
      for (int j = 0; j < V; j += 2)
        if (i + j < dims) {
          const float2 t = angle[(i + j) / 2];
          const float u = a[j], v = a[j + 1];
          a[j] = u * t.x - v * t.y;
          a[j + 1] = v * t.x + u * t.y;
        }
      return;
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const int c = i + j;
    if (c >= dims) break;
    const bool low = interleaved ? c % 2 == 0 : c < half;
    const float other = column(interleaved ? (low ? c + 1 : c - 1) : low ? c + half : c - half);
    const float2 t = angle[interleaved ? c / 2 : low ? c : c - half];
    a[j] = low ? a[j] * t.x - other * t.y : a[j] * t.x + other * t.y;
  }
}

// One group of LG lanes per (token, head); heads [0, H) queries, then G keys, then G values (G 0: queries alone).  Queries and keys pass an RMS norm
// where they have a weight or `unit` asks for it (a rotation keeps a head's square sum, so one without a weight may stand before or behind it).
template <typename T, int V, int LG>
__global__ void __launch_bounds__(256)
head_norm_append_kernel(const T* __restrict__ qkv, long long row_stride, const T* __restrict__ bias, const T* __restrict__ qw, const T* __restrict__ kw,
                        float eps, int unit, Turn turn, const int* __restrict__ positions, long long items, int S, int H, int G, int dk, int dv, int D,
                        T* __restrict__ packed, T* __restrict__ kpool, T* __restrict__ vpool, Pool pool) {
  const unsigned item = blockIdx.x * (256 / LG) + threadIdx.x / LG;
  const int lane = threadIdx.x % LG;
  const bool on = item < items;                      // every lane stays for the sums
  const unsigned heads = H + 2 * G, tt = on ? item / heads : 0;
  const long long t = tt;
  const int h = on ? static_cast<int>(item - tt * heads) : 0;
  const int part = h < H ? 0 : h < H + G ? 1 : 2, width = part == 2 ? dv : dk;
  const int at = part == 2 ? (H + G) * dk + (h - H - G) * dv : h * dk;
  const T* src = qkv + t * row_stride + at;
  const T* b = bias == nullptr ? nullptr : bias + at;
  const T* w = part == 0 ? qw : part == 1 ? kw : nullptr;
  const bool normed = part != 2 && (w != nullptr || unit);
  const int pos = part != 0 ? positions[t] : -1;
  float ss = 0.f;
  if (normed) {
    for (int i = lane * V; i < width; i += LG * V) {
      float a[V];
      load_v<V>(src + i, a);
      if (b != nullptr) {
        float c[V];
        load_v<V>(b + i, c);
#pragma unroll
        for (int j = 0; j < V; ++j) a[j] += c[j];
      }
#pragma unroll
      for (int j = 0; j < V; ++j) ss += a[j] * a[j];
    }
  }
#pragma unroll
  for (int o = LG / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!on) return;
  const float r = normed ? 1.f / sqrtf(ss / width + eps) : 1.f;
  const float2* angle = part != 2 && turn.table != nullptr ? turn.table + t * (turn.dims / 2) : nullptr;
  T* dst = packed + static_cast<long long>(item) * D;
  T* to_pool = nullptr;
  if (pos >= 0) {
    const long long tok = pool_token(pool, static_cast<int>(tt / static_cast<unsigned>(S)), pos);
    to_pool = (part == 1 ? kpool : vpool) + (tok * G + (part == 1 ? h - H : h - H - G)) * D;
  }
  for (int i = lane * V; i < D; i += LG * V) {
    float a[V];
    if (i < width) {
      head_columns<T, V>(src, b, w, r, i, angle, turn.dims, turn.interleaved, a);
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] = 0.f;
    }
    store_v<V>(dst + i, a);
    if (to_pool != nullptr) store_v<V>(to_pool + i, a);
  }
}

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// grid (tokens, ceil(H dv / (256 V))): out [tokens, H, dv] = o [tokens, H, D] * sigmoid(gate [tokens, *] of the head)
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_gate_kernel(const T* __restrict__ o, const T* __restrict__ gate, long long gate_stride, T* __restrict__ out, int H, int dv, int D) {
  const int i = (blockIdx.y * 256 + threadIdx.x) * V;
  if (i >= H * dv) return;
  const long long t = blockIdx.x;
  const int h = i / dv;
  float a[V];
  load_v<V>(o + (t * H + h) * D + (i - h * dv), a);
  const float s = sigmoid(ld(gate + t * gate_stride + h));
#pragma unroll
  for (int j = 0; j < V; ++j) a[j] *= s;
  store_v<V>(out + t * H * dv + i, a);
}

// What a layer's attention adds to the causal softmax: each part off at 0 / null.
template <typename T>
struct Extras {
  int chunk;               // a query sees no key from before the start of its chunk
  int window, keep;        // a query sees its last `window` keys (its own among them) and the row's first `keep`
  float cap;               // scores become cap tanh(score / cap); the tensor-core form holds it in the log2 domain
  const float* sinks;      // [H]: joins the denominator, has no value
  const T* gate;           // [tokens, *]: head h's output times sigmoid(gate[token, h])
  long long gate_stride;
  const float* gain;       // [H]: the head's scores times it, in front of the cap
  const float* sig;        // [H]: weights are sigmoid(score + sig[head]) instead of the softmax
};

// First key a query sees, the kept ones aside.
template <typename T>
__device__ __forceinline__ int first_seen(int pos, const Extras<T>& ex) {
  if (pos <= 0) return 0;
  const int start = ex.chunk > 0 ? pos / ex.chunk * ex.chunk : 0;
  return ex.window > 0 ? max(start, pos - ex.window + 1) : start;
}

constexpr int BQ = 32, BK = 32, THREADS = 256, WIDE = 576;

__host__ __device__ inline int key_piece(int dk) { return dk <= WIDE ? dk : 256; }

// grid (query tiles, G, rows).  q [R, S, *, D] with a token stride; out [R, S, H, dv] contiguous.  NJ: value columns per thread / 4.
template <typename T, int NJ>
__global__ void __launch_bounds__(THREADS)
paged_attend_kernel(const T* __restrict__ q, long long q_token_stride, const T* __restrict__ kpool, const T* __restrict__ vpool,
                    const int* __restrict__ positions, int S, int H, int G, int dk, int dv, int D, float scale, T* __restrict__ out, Pool pool,
                    Extras<T> ex) {
  extern __shared__ __align__(16) float smem[];
  // keys past WIDE columns go through shared memory (with their queries) in pieces; values past a block's columns are other blocks' work
  const int kc = key_piece(dk), kst = ((kc + 3) & ~3) + 4, vst = NJ * 32 + 4;
  float* sq = smem;                     // [BQ][kst]
  float* sk = sq + BQ * kst;            // [BK][kst]
  float* sv = sk + BK * kst;            // [BK][vst]
  float* sp = sv + BK * vst;            // [BQ][BK + 1]
  __shared__ int s_pos[BQ];
  __shared__ long long s_tok[BK];
  const int parts = (dv + NJ * 32 - 1) / (NJ * 32), row = blockIdx.z, g = blockIdx.y / parts, v0 = (blockIdx.y - g * parts) * NJ * 32, Gq = H / G;
  const int r0 = blockIdx.x * BQ, rows = S * Gq;
  const int tid = threadIdx.x;
  if (tid < BQ) {
    const int r = r0 + tid;
    s_pos[tid] = r < rows ? positions[static_cast<long long>(row) * S + r / Gq] : -1;
  }
  __syncthreads();
  int last = -1, lowest = INT_MAX;
  for (int i = 0; i < BQ; ++i) {
    last = max(last, s_pos[i]);
    if (s_pos[i] >= 0) lowest = min(lowest, first_seen(s_pos[i], ex));
  }
  auto load_queries = [&](int c0) {
    for (int i = tid; i < BQ * kst; i += THREADS) {
      const int r = i / kst, c = i - r * kst;
      float v = 0.f;
      if (c < kc && c0 + c < dk && s_pos[r] >= 0) {
        const int gr = r0 + r;
        const int head = g * Gq + gr % Gq;
        v = ld(q + (static_cast<long long>(row) * S + gr / Gq) * q_token_stride + static_cast<long long>(head) * D + c0 + c) *
            (ex.gain != nullptr ? scale * ex.gain[head] : scale);
      }
      sq[i] = v;
    }
  };
  if (kc == dk) load_queries(0);
  const int qr = tid >> 3, ql = tid & 7;
  const int my_pos = s_pos[qr], my_first = first_seen(my_pos, ex);
  const float my_sig = ex.sig != nullptr ? ex.sig[g * Gq + (r0 + qr) % Gq] : 0.f;
  float m = -INFINITY, l = 0.f, acc[NJ][4];
#pragma unroll
  for (int j = 0; j < NJ; ++j) { acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f; }
  // the tiles of the kept first keys, then those from the lowest first key on
  const int lo = last < 0 ? 0 : lowest / BK, kept = last < 0 ? 0 : min((ex.keep + BK - 1) / BK, lo), tiles = kept + (last + BK) / BK - lo;
  for (int t = 0; t < tiles; ++t) {
    const int k0 = (t < kept ? t : lo + t - kept) * BK;
    __syncthreads();
    if (tid < BK) s_tok[tid] = k0 + tid <= last ? pool_token(pool, row, k0 + tid) : -1;
    __syncthreads();
    for (int i = tid; i < BK * vst; i += THREADS) {
      const int r = i / vst, c = i - r * vst;
      sv[i] = (v0 + c < dv && s_tok[r] >= 0) ? ld(vpool + (s_tok[r] * G + g) * D + v0 + c) : 0.f;
    }
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    for (int c0 = 0; c0 < dk; c0 += kc) {
      if (kc != dk) {
        if (c0 > 0) __syncthreads();                 // the piece before has been read
        load_queries(c0);
      }
      for (int i = tid; i < BK * kst; i += THREADS) {
        const int r = i / kst, c = i - r * kst;
        sk[i] = (c < kc && c0 + c < dk && s_tok[r] >= 0) ? ld(kpool + (s_tok[r] * G + g) * D + c0 + c) : 0.f;
      }
      __syncthreads();
      for (int c = 0; c < kst - 4; c += 4) {
        const float4 a = *reinterpret_cast<const float4*>(sq + qr * kst + c);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float4 b = *reinterpret_cast<const float4*>(sk + (ql + 8 * j) * kst + c);
          s[j] += a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w;
        }
      }
    }
    float bm = -INFINITY;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (ex.cap > 0.f) s[j] = ex.cap * tanhf(s[j] / ex.cap);
      const int key = k0 + ql + 8 * j;
      if (key > my_pos || (key < my_first && key >= ex.keep)) s[j] = -INFINITY;
      bm = fmaxf(bm, s[j]);
    }
    if (ex.sig != nullptr) {
#pragma unroll
      for (int j = 0; j < 4; ++j) sp[qr * (BK + 1) + ql + 8 * j] = s[j] == -INFINITY ? 0.f : sigmoid(s[j] + my_sig);
      l = 1.f;                                       // nothing to divide by
      __syncwarp();
    } else {
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, o));
      const float mn = fmaxf(m, bm);
      const float alpha = m == -INFINITY ? 0.f : expf(m - mn);
      float ps = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float p = s[j] == -INFINITY ? 0.f : expf(s[j] - mn);
        ps += p;
        sp[qr * (BK + 1) + ql + 8 * j] = p;
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
      l = l * alpha + ps;
      m = mn;
      __syncwarp();
#pragma unroll
      for (int j = 0; j < NJ; ++j) { acc[j][0] *= alpha; acc[j][1] *= alpha; acc[j][2] *= alpha; acc[j][3] *= alpha; }
    }
    for (int k = 0; k < BK; ++k) {
      const float p = sp[qr * (BK + 1) + k];
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const float4 v = *reinterpret_cast<const float4*>(sv + k * vst + ql * 4 + 32 * j);
        acc[j][0] += p * v.x; acc[j][1] += p * v.y; acc[j][2] += p * v.z; acc[j][3] += p * v.w;
      }
    }
  }
  const int gr = r0 + qr;
  if (gr >= rows) return;
  float inv = l > 0.f ? 1.f / l : 0.f;
  const int head = g * Gq + gr % Gq;
  if (ex.sinks != nullptr && l > 0.f) {
    const float sink = ex.sinks[head], top = fmaxf(m, sink), f = expf(m - top);
    inv = f / (l * f + expf(sink - top));
  }
  if (ex.gate != nullptr) inv *= sigmoid(ld(ex.gate + (static_cast<long long>(row) * S + gr / Gq) * ex.gate_stride + head));
  T* o = out + ((static_cast<long long>(row) * S + gr / Gq) * H + g * Gq + gr % Gq) * dv;
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = v0 + ql * 4 + 32 * j + e;
      if (c < dv) st(o + c, acc[j][e] * inv);
    }
}

// ---- tensor-core form: 64 rows of work a CTA (4 warps of 16), key / value tiles of 64 through a two-stage cp.async ring, online softmax in
// the log2 domain with fp32 scores and sums, probabilities in bf16 for the value product.
constexpr int MQ = 64, MK = 64, MTHREADS = 128;

__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool live) {
  const int n = live ? 16 : 0;                     // 0: the 16 bytes are filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

// tanh to fp32 accuracy relative to 1
__device__ __forceinline__ float soft_tanh(float x) { return 1.f - __fdividef(2.f, 1.f + exp2f(x * 2.8853900817779268f)); }

// SIG: sigmoid weights
template <int D, bool SIG>
__global__ void __launch_bounds__(MTHREADS)
paged_attend_mma_kernel(const bf16* __restrict__ q, long long q_token_stride, const bf16* __restrict__ kpool, const bf16* __restrict__ vpool,
                        const int* __restrict__ positions, int S, int H, int G, int dv, float scale_log2, bf16* __restrict__ out, Pool pool,
                        Extras<bf16> ex) {
  using namespace mma16;
  constexpr int ST = D + 8;                        // smem row stride
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* sq = reinterpret_cast<bf16*>(raw);         // [MQ][ST]
  bf16* sk = sq + MQ * ST;                         // [2][MK][ST]
  bf16* sv = sk + 2 * MK * ST;                     // [2][MK][ST]
  __shared__ int s_pos[MQ];
  const int row = blockIdx.z, g = blockIdx.y, Gq = H / G;
  const int r0 = blockIdx.x * MQ, rows = S * Gq;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid < MQ) {
    const int r = r0 + tid;
    s_pos[tid] = r < rows ? positions[static_cast<long long>(row) * S + r / Gq] : -1;
  }
  __syncthreads();
  int last = -1, lowest = INT_MAX;
  for (int i = 0; i < MQ; ++i) {
    last = max(last, s_pos[i]);
    if (s_pos[i] >= 0) lowest = min(lowest, first_seen(s_pos[i], ex));
  }
  // the tiles of the kept first keys, then those from the lowest first key on
  const int lo = last < 0 ? 0 : lowest / MK, kept = last < 0 ? 0 : min((ex.keep + MK - 1) / MK, lo), tiles = kept + (last + MK) / MK - lo;
  auto first_key_of = [&](int t) { return (t < kept ? t : lo + t - kept) * MK; };
  for (int i = tid; i < MQ * (D / 8); i += MTHREADS) {
    const int r = i / (D / 8), c = (i % (D / 8)) * 8, gr = r0 + r;
    const bool live = s_pos[r] >= 0;
    const bf16* src = live ? q + (static_cast<long long>(row) * S + gr / Gq) * q_token_stride + static_cast<long long>(g * Gq + gr % Gq) * D + c : q;
    cp16(smem_addr(sq + r * ST + c), src, live);
  }
  auto fetch = [&](int t) {
    bf16* dk_ = sk + (t & 1) * MK * ST;
    bf16* dv_ = sv + (t & 1) * MK * ST;
    const int k0 = first_key_of(t);
    for (int i = tid; i < MK * (D / 8); i += MTHREADS) {
      const int r = i / (D / 8), c = (i % (D / 8)) * 8, key = k0 + r;
      const bool live = key <= last;
      const long long off = live ? (pool_token(pool, row, key) * G + g) * D + c : 0;
      cp16(smem_addr(dk_ + r * ST + c), kpool + off, live);
      cp16(smem_addr(dv_ + r * ST + c), vpool + off, live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int lg = lane >> 2, t2 = (lane & 3) * 2;
  const int p0 = s_pos[warp * 16 + lg], p1 = s_pos[warp * 16 + lg + 8];
  const int f0_ = first_seen(p0, ex), f1_ = first_seen(p1, ex);        // first keys the rows see
  const int h0_ = g * Gq + (r0 + warp * 16 + lg) % Gq, h1_ = g * Gq + (r0 + warp * 16 + lg + 8) % Gq;
  const float c0_ = ex.gain != nullptr ? scale_log2 * ex.gain[h0_] : scale_log2, c1_ = ex.gain != nullptr ? scale_log2 * ex.gain[h1_] : scale_log2;
  const float b0_ = SIG ? ex.sig[h0_] * 1.4426950408889634f : 0.f, b1_ = SIG ? ex.sig[h1_] * 1.4426950408889634f : 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f, o[D / 8][4];
#pragma unroll
  for (int j = 0; j < D / 8; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  if (tiles > 0) fetch(0);
  for (int t = 0; t < tiles; ++t) {
    if (t + 1 < tiles) {
      fetch(t + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const bf16* tk = sk + (t & 1) * MK * ST;
    const bf16* tv = sv + (t & 1) * MK * ST;
    float s[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) { s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f; }
#pragma unroll
    for (int kk = 0; kk < D; kk += 16) {
      uint32_t a[4];
      ldsm4(a, smem_addr(sq + (warp * 16 + (lane & 15)) * ST + kk + (lane >> 4) * 8));
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint32_t b[4];
        ldsm4(b, smem_addr(tk + (j * 16 + (lane & 7) + (lane >> 4) * 8) * ST + kk + ((lane >> 3) & 1) * 8));
        mma(s[2 * j], a, b[0], b[1]);
        mma(s[2 * j + 1], a, b[2], b[3]);
      }
    }
    float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int key = first_key_of(t) + j * 8 + t2;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = s[j][e] * (e < 2 ? c0_ : c1_);
        if (ex.cap > 0.f) v = ex.cap * soft_tanh(v / ex.cap);
        const int at = key + (e & 1), p = e < 2 ? p0 : p1, f = e < 2 ? f0_ : f1_;
        const bool seen = at <= p && (at >= f || at < ex.keep);
        if (SIG) s[j][e] = seen ? __fdividef(1.f, 1.f + exp2f(-(v + (e < 2 ? b0_ : b1_)))) : 0.f;
        else s[j][e] = seen ? v : -INFINITY;
      }
      x0 = fmaxf(x0, fmaxf(s[j][0], s[j][1]));
      x1 = fmaxf(x1, fmaxf(s[j][2], s[j][3]));
    }
    if constexpr (!SIG) {
#pragma unroll
    for (int d = 1; d < 4; d <<= 1) {
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, d));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, d));
    }
    const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);
    const float b0 = n0 == -INFINITY ? 0.f : n0, b1 = n1 == -INFINITY ? 0.f : n1;      // a row that has seen nothing yet
    const float f0 = exp2f(m0 - b0), f1 = exp2f(m1 - b1);
    m0 = n0; m1 = n1;
    l0 *= f0; l1 *= f1;
#pragma unroll
    for (int j = 0; j < D / 8; ++j) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      s[j][0] = exp2f(s[j][0] - b0); s[j][1] = exp2f(s[j][1] - b0);
      s[j][2] = exp2f(s[j][2] - b1); s[j][3] = exp2f(s[j][3] - b1);
      l0 += s[j][0] + s[j][1];
      l1 += s[j][2] + s[j][3];
    }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const uint32_t a[4] = {pack2(s[2 * j][0], s[2 * j][1]), pack2(s[2 * j][2], s[2 * j][3]), pack2(s[2 * j + 1][0], s[2 * j + 1][1]),
                             pack2(s[2 * j + 1][2], s[2 * j + 1][3])};
#pragma unroll
      for (int n = 0; n < D / 16; ++n) {
        uint32_t b[4];
        ldsm4_t(b, smem_addr(tv + (j * 16 + (lane & 15)) * ST + n * 16 + (lane >> 4) * 8));
        mma(o[2 * n], a, b[0], b[1]);
        mma(o[2 * n + 1], a, b[2], b[3]);
      }
    }
    __syncthreads();                               // the tile's stage is refilled two tiles on
  }
#pragma unroll
  for (int d = 1; d < 4; d <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, d);
    l1 += __shfl_xor_sync(0xffffffffu, l1, d);
  }
  const float i0 = SIG ? 1.f : l0 > 0.f ? 1.f / l0 : 0.f, i1 = SIG ? 1.f : l1 > 0.f ? 1.f / l1 : 0.f;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int gr = r0 + warp * 16 + lg + 8 * e;
    if (gr >= rows) continue;
    float inv = e ? i1 : i0;
    const int head = g * Gq + gr % Gq;
    if (ex.sinks != nullptr && inv > 0.f) {
      const float m = e ? m1 : m0, l = e ? l1 : l0, sink = ex.sinks[head] * 1.4426950408889634f, top = fmaxf(m, sink), f = exp2f(m - top);
      inv = f / (l * f + exp2f(sink - top));
    }
    if (ex.gate != nullptr) inv *= sigmoid(ld(ex.gate + (static_cast<long long>(row) * S + gr / Gq) * ex.gate_stride + head));
    bf16* dst = out + ((static_cast<long long>(row) * S + gr / Gq) * H + g * Gq + gr % Gq) * dv;
#pragma unroll
    for (int j = 0; j < D / 8; ++j) {
      const int c = j * 8 + t2;
      if (c < dv) dst[c] = __float2bfloat16(o[j][2 * e] * inv);
      if (c + 1 < dv) dst[c + 1] = __float2bfloat16(o[j][2 * e + 1] * inv);
    }
  }
}

template <int D, bool SIG>
int attend_mma(const bf16* q, long long qs, const bf16* kpool, const bf16* vpool, const int* positions, int R, int S, int H, int G, int dv, float scale,
               bf16* out, const Pool& pool, const Extras<bf16>& ex, cudaStream_t stream) {
  const int smem = (MQ + 4 * MK) * (D + 8) * 2;
  cudaError_t e = cudaFuncSetAttribute(paged_attend_mma_kernel<D, SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  const long long tiles = (static_cast<long long>(S) * (H / G) + MQ - 1) / MQ;
  paged_attend_mma_kernel<D, SIG><<<dim3(static_cast<unsigned>(tiles), G, R), MTHREADS, smem, stream>>>(q, qs, kpool, vpool, positions, S, H, G, dv,
                                                                                              scale * 1.4426950408889634f, out, pool, ex);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int NJ>
int attend(const T* q, long long qs, const T* kpool, const T* vpool, const int* positions, int R, int S, int H, int G, int dk, int dv, int D,
           float scale, T* out, const Pool& pool, const Extras<T>& ex, cudaStream_t stream) {
  const int kst = ((key_piece(dk) + 3) & ~3) + 4, vst = NJ * 32 + 4, parts = (dv + NJ * 32 - 1) / (NJ * 32);
  const size_t smem = static_cast<size_t>(BQ * kst + BK * kst + BK * vst + BQ * (BK + 1)) * 4;
  if (smem > 225 * 1024) return -3;
  cudaError_t e = cudaFuncSetAttribute(paged_attend_kernel<T, NJ>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const long long tiles = (static_cast<long long>(S) * (H / G) + BQ - 1) / BQ;
  paged_attend_kernel<T, NJ><<<dim3(static_cast<unsigned>(tiles), G * parts, R), THREADS, smem, stream>>>(q, qs, kpool, vpool, positions, S, H, G, dk, dv, D, scale, out,
                                                                                             pool, ex);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int attend_any(const void* q, long long qs, const void* kpool, const void* vpool, const int* positions, int R, int S, int H, int G, int dk, int dv,
               int D, float scale, void* out, const Pool& pool, int chunk, int window, int keep, float softcap, const float* sinks, const void* gate,
               long long gate_stride, const float* gain, const float* sig, cudaStream_t stream) {
  const Extras<T> ex{chunk, window, keep, softcap, sinks, static_cast<const T*>(gate), gate_stride, gain, sig};
#define DEWB_ATTEND(NN) attend<T, NN>(static_cast<const T*>(q), qs, static_cast<const T*>(kpool), static_cast<const T*>(vpool), positions, R, S, H, G, \
                                      dk, dv, D, scale, static_cast<T*>(out), pool, ex, stream)
  const int nj = (dv + 31) / 32;
  if (nj <= 1) return DEWB_ATTEND(1);
  if (nj <= 2) return DEWB_ATTEND(2);
  if (nj <= 4) return DEWB_ATTEND(4);
  if (nj <= 8) return DEWB_ATTEND(8);
  if (nj <= 16) return DEWB_ATTEND(16);
  return DEWB_ATTEND(8);
#undef DEWB_ATTEND
}

}  // namespace paged
}  // namespace dewb

using namespace dewb::paged;

// qkv [R * S, H dk + G dk + G dv] -> packed [R * S, H + 2 G, D] and the pools [*, page_size, G, D].  `every` 0: no temperature.
extern "C" int dewb_qk_norm_append(const void* qkv, const void* qw, const void* kw, float eps, float coef, int every, const int* positions, int R,
                                   int S, int H, int G, int dk, int dv, int D, void* packed, void* kpool, void* vpool, const int* page_table,
                                   int page_size, int max_pages, const int* row_ids, int fp32, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (H < 1 || G < 1 || H % G || dk < 1 || dv < 1 || D < dk || D < dv || page_size < 1 || max_pages < 1 || every < 0) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Pool pool{page_table, page_size, max_pages, row_ids};
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && D % 4 == 0 && aligned(qkv, 16) && aligned(qw, 16) && aligned(kw, 16) && aligned(packed, 16) &&
                   aligned(kpool, 16) && aligned(vpool, 16);
  const dim3 grid(static_cast<unsigned>(R) * static_cast<unsigned>(S), 3);
#define DEWB_PREP(TT, VV) qk_norm_append_kernel<TT, VV><<<grid, PREP_THREADS, 0, stream>>>(static_cast<const TT*>(qkv), static_cast<const TT*>(qw), \
    static_cast<const TT*>(kw), eps, coef, every, positions, S, H, G, dk, dv, D, static_cast<TT*>(packed), static_cast<TT*>(kpool), \
    static_cast<TT*>(vpool), pool)
  if (fp32) { if (vec) DEWB_PREP(float, 4); else DEWB_PREP(float, 1); }
  else { if (vec && dk % 8 == 0 && dv % 8 == 0 && D % 8 == 0) DEWB_PREP(bf16, 8); else if (vec) DEWB_PREP(bf16, 4); else DEWB_PREP(bf16, 1); }
#undef DEWB_PREP
  return static_cast<int>(cudaGetLastError());
}

// qkv [R * S, row_stride >= H dk + G dk + G dv] -> packed [R * S, H + 2 G, D] and the pools; per-head norms with the weights qw, kw [dk] (null: none;
// `unit`: a norm without a weight), bias [H dk + G dk + G dv] (null: none); `table` [R * S, dims / 2, 2] (null: no rotation) turns the first `dims`
// columns of the query and key heads.  G 0: a layer without keys and values of its own (the pools are not touched).
extern "C" int dewb_head_norm_append(const void* qkv, long long row_stride, const void* bias, const void* qw, const void* kw, float eps, int unit,
                                     const float* table, int dims, int interleaved, const int* positions, int R, int S, int H, int G, int dk, int dv,
                                     int D, void* packed, void* kpool, void* vpool, const int* page_table, int page_size, int max_pages,
                                     const int* row_ids, int fp32, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (H < 1 || G < 0 || (G > 0 && H % G) || dk < 1 || dv < 1 || D < dk || D < dv || page_size < 1 || max_pages < 1 ||
      row_stride < static_cast<long long>(H + G) * dk + static_cast<long long>(G) * dv || (table != nullptr && (dims < 2 || dims % 2 || dims > dk)))
    return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Pool pool{page_table, page_size, max_pages, row_ids};
  const Turn turn{reinterpret_cast<const float2*>(table), table == nullptr ? 0 : dims, interleaved};
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && D % 4 == 0 && row_stride % 4 == 0 && aligned(qkv, 16) && aligned(bias, 16) && aligned(qw, 16) &&
                   aligned(kw, 16) && aligned(packed, 16) && aligned(kpool, 16) && aligned(vpool, 16);
  const long long items = static_cast<long long>(R) * S * (H + 2 * G);
  const bool vec8 = vec && !fp32 && dk % 8 == 0 && dv % 8 == 0 && D % 8 == 0 && row_stride % 8 == 0;
  const int v = vec8 ? 8 : vec ? 4 : 1, lg = D <= 8 * v ? 8 : D <= 16 * v ? 16 : 32;
  const long long blocks = (items * lg + 255) / 256;
  if (items > 0x7fffffffll) return -3;
#define DEWB_HEADS(TT, VV, LL) head_norm_append_kernel<TT, VV, LL><<<static_cast<unsigned>(blocks), 256, 0, stream>>>(static_cast<const TT*>(qkv), \
    row_stride, static_cast<const TT*>(bias), static_cast<const TT*>(qw), static_cast<const TT*>(kw), eps, unit, turn, positions, items, S, H, G, dk, dv, D, \
    static_cast<TT*>(packed), static_cast<TT*>(kpool), static_cast<TT*>(vpool), pool)
#define DEWB_HEADS_L(TT, VV) do { if (lg == 8) DEWB_HEADS(TT, VV, 8); else if (lg == 16) DEWB_HEADS(TT, VV, 16); else DEWB_HEADS(TT, VV, 32); } while (0)
  if (fp32) { if (vec) DEWB_HEADS_L(float, 4); else DEWB_HEADS_L(float, 1); }
  else { if (vec8) DEWB_HEADS_L(bf16, 8); else if (vec) DEWB_HEADS_L(bf16, 4); else DEWB_HEADS_L(bf16, 1); }
#undef DEWB_HEADS_L
#undef DEWB_HEADS
  return static_cast<int>(cudaGetLastError());
}

// o [tokens, H, D] -> out [tokens, H, dv], each head times sigmoid(gate[token * gate_stride + head])
extern "C" int dewb_head_gate(const void* o, const void* gate, long long gate_stride, void* out, long long tokens, int H, int dv, int D, int fp32,
                              void* stream_ptr) {
  if (tokens <= 0) return 0;
  if (H < 1 || dv < 1 || D < dv || gate_stride < H || gate == nullptr) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bool vec = dv % 4 == 0 && D % 4 == 0 && aligned(o, 16) && aligned(out, 16);
  const int v = vec && !fp32 && dv % 8 == 0 && D % 8 == 0 ? 8 : vec ? 4 : 1;
  const int blocks = (H * dv + 256 * v - 1) / (256 * v);
  if (blocks > 65535) return -3;
  const dim3 grid(static_cast<unsigned>(tokens), blocks);
#define DEWB_GATE(TT, VV) head_gate_kernel<TT, VV><<<grid, 256, 0, stream>>>(static_cast<const TT*>(o), static_cast<const TT*>(gate), gate_stride,     static_cast<TT*>(out), H, dv, D)
  if (fp32) { if (v == 4) DEWB_GATE(float, 4); else DEWB_GATE(float, 1); }
  else { if (v == 8) DEWB_GATE(bf16, 8); else if (v == 4) DEWB_GATE(bf16, 4); else DEWB_GATE(bf16, 1); }
#undef DEWB_GATE
  return static_cast<int>(cudaGetLastError());
}

// positions [n] (below 0: taken as 0), frequency [half] -> out [n, half, 2]
extern "C" int dewb_rotary_angles(const int* positions, const double* frequency, float* out, long long n, int half, void* stream_ptr) {
  if (n <= 0) return 0;
  const long long blocks = (n * half + 255) / 256;
  if (half < 1 || blocks > 0x7fffffffll) return -3;
  rotary_angles_kernel<<<static_cast<unsigned>(blocks), 256, 0, reinterpret_cast<cudaStream_t>(stream_ptr)>>>(positions, frequency, reinterpret_cast<float2*>(out),
                                                                                                              n, half);
  return static_cast<int>(cudaGetLastError());
}

static bool range_ok(int chunk, int window, int keep, float softcap) {
  return chunk >= 0 && window >= 0 && keep >= 0 && (keep == 0 || chunk == 0) && softcap >= 0.f;
}

// `chunk` 0, `window` 0 (and `keep` with it), `softcap` 0, `sinks`, `gate`, `gain` and `sig` null: off (see Extras).
extern "C" int dewb_paged_attend(const void* q, long long q_token_stride, const void* kpool, const void* vpool, const int* positions, int R, int S,
                                 int H, int G, int dk, int dv, int D, float scale, int chunk, int window, int keep, float softcap, const float* sinks, const void* gate,
                                 long long gate_stride, const float* gain, const float* sig, void* out, const int* page_table, int page_size, int max_pages,
                                 const int* row_ids, int fp32, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (H < 1 || G < 1 || H % G || dk < 1 || dv < 1 || D < dk || D < dv || page_size < 1 || max_pages < 1 || !range_ok(chunk, window, keep, softcap) || (sig != nullptr && sinks != nullptr)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Pool pool{page_table, page_size, max_pages, row_ids};
  if (fp32) return attend_any<float>(q, q_token_stride, kpool, vpool, positions, R, S, H, G, dk, dv, D, scale, out, pool, chunk, window, keep, softcap, sinks, gate, gate_stride, gain, sig, stream);
  return attend_any<bf16>(q, q_token_stride, kpool, vpool, positions, R, S, H, G, dk, dv, D, scale, out, pool, chunk, window, keep, softcap, sinks, gate, gate_stride, gain, sig, stream);
}

// The tensor-core form (bf16; pools D = 64, 128 or 256 wide; q on 16-byte boundaries with a token stride of a multiple of 8).
extern "C" int dewb_paged_attend_mma(const void* q, long long q_token_stride, const void* kpool, const void* vpool, const int* positions, int R, int S,
                                     int H, int G, int dv, int D, float scale, int chunk, int window, int keep, float softcap, const float* sinks, const void* gate, long long gate_stride,
                                     const float* gain, const float* sig, void* out, const int* page_table, int page_size, int max_pages, const int* row_ids, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (H < 1 || G < 1 || H % G || dv < 1 || D < dv || page_size < 1 || max_pages < 1 || !range_ok(chunk, window, keep, softcap) || (sig != nullptr && sinks != nullptr) ||
      q_token_stride % 8 || !aligned(q, 16) || !aligned(kpool, 16) ||
      !aligned(vpool, 16))
    return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Pool pool{page_table, page_size, max_pages, row_ids};
  const bf16 *qp = static_cast<const bf16*>(q), *kp = static_cast<const bf16*>(kpool), *vp = static_cast<const bf16*>(vpool);
  bf16* op = static_cast<bf16*>(out);
  const Extras<bf16> ex{chunk, window, keep, softcap * 1.4426950408889634f, sinks, static_cast<const bf16*>(gate), gate_stride, gain, sig};
#define DEWB_MMA(DD, SS) attend_mma<DD, SS>(qp, q_token_stride, kp, vp, positions, R, S, H, G, dv, scale, op, pool, ex, stream)
  if (D == 64) return sig != nullptr ? DEWB_MMA(64, true) : DEWB_MMA(64, false);
  if (D == 128) return sig != nullptr ? DEWB_MMA(128, true) : DEWB_MMA(128, false);
  if (D == 256) return sig != nullptr ? DEWB_MMA(256, true) : DEWB_MMA(256, false);
#undef DEWB_MMA
  return -3;
}
