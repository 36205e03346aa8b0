// Row kernels of decoders whose residual is a bundle of fp32 streams, for sm_100a.  All are bandwidth bound: one pass over the operands,
// 16-byte accesses, fp32 arithmetic.
//
//   embed_streams   H[t, s, :] = gain * embed[token t] (+ pos[position t]) for every stream s
//   stream_step     one residual step between two sub-layers: the pending write of the sub-layer that just ran
//                       H'[t] = sum_s mix[s, t] H[s] + out[t] * (gain scale . y + gain2 scale2 . y2)
//                   (in place), the read of the next one, u = sum_s read[s] H'[s], and its norm (layer norm without a bias, or RMS norm,
//                   whose weights may be stored as their distance from `around`); y may pass an RMS norm of its own first (a block that
//                   normalises what its sub-layers return); y2 is there when two sub-layers read the same norm and join together.  Without connection
//                   weights the streams keep themselves and take y as it is: one such stream is the ordinary fp32 residual, which has a
//                   form of its own (residual_step).  What else joins the one stream on the way (Join): the token's embedding again, and a vector
//                   (a looped block of layers takes them in front of each pass).  The norm's weight may be one number for all coordinates.
//   clamped_glu     g sigmoid(alpha g) (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit)
//   gelu_glu        gelu(gate) up, the tanh form of gelu
//   sigmoid_gated_norm   RMS norm over a whole row times a weight times sigmoid(gate)
//   softcap         cap tanh(x / cap), fp32 out (logits)
//
// Activations are bf16 or fp32 (template T); the streams, the connection weights and every sum are fp32.  Compiled without fast math.
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/rows.cuh"

namespace dewb {
namespace streams {

using namespace rows;
constexpr int MAX_STREAMS = 16;
constexpr int THREADS = 256;

template <typename T, int V>
__global__ void __launch_bounds__(THREADS)
embed_streams_kernel(const long long* __restrict__ tokens, const int* __restrict__ positions, const T* __restrict__ embed,
                     const T* __restrict__ pos, float* __restrict__ H, int n, int d, int vocab, int max_pos, float gain) {
  const long long t = blockIdx.x;
  const long long tok = min(max(tokens[t], 0ll), static_cast<long long>(vocab - 1));
  const int p = min(max(positions == nullptr ? 0 : positions[t], 0), max_pos - 1);
  for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
    float a[V];
    load_v<V>(embed + tok * d + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] *= gain;
    if (pos != nullptr) {
      float b[V];
      load_v<V>(pos + static_cast<long long>(p) * d + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] += b[j];
    }
    for (int s = 0; s < n; ++s) store_v<V>(H + (t * n + s) * d + i, a);
  }
}

// What joins the residual beside the sub-layers: add [d] and gain * table[token] (null: neither).
template <typename T>
struct Join {
  const T* add;
  const T* table;
  const long long* tokens;
  int vocab;
  float gain;
  __host__ __device__ __forceinline__ bool any() const { return add != nullptr || table != nullptr; }
  template <int V>
  __device__ __forceinline__ void to(float (&x)[V], long long t, int i, int d) const {
    if (table != nullptr) {
      float e[V];
      load_v<V>(table + min(max(tokens[t], 0ll), static_cast<long long>(vocab - 1)) * d + i, e);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] += gain * e[j];
    }
    if (add != nullptr) {
      float e[V];
      load_v<V>(add + i, e);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] += e[j];
    }
  }
};

// V weights of a norm: `one` - the same number for every coordinate
template <typename T, int V>
__device__ __forceinline__ void load_weight(const T* w, int one, int i, float (&c)[V]) {
  if (one) {
    float x[1];
    load_v<1>(w, x);
#pragma unroll
    for (int j = 0; j < V; ++j) c[j] = x[0];
  } else {
    load_v<V>(w + i, c);
  }
}

// NS: the number of streams when it is small and known (registers sized for it), 0: any number up to MAX_STREAMS.
template <typename T, int V, int NS>
__global__ void __launch_bounds__(THREADS)
stream_step_kernel(float* __restrict__ H, const T* __restrict__ y, const T* __restrict__ y_weight, const T* __restrict__ scale,
                   const float* __restrict__ mix, const float* __restrict__ out, const float* __restrict__ read, const T* __restrict__ w,
                   T* __restrict__ normed, int n_rt, int d, float y_eps, float eps, int rms, const T* __restrict__ y2, const T* __restrict__ scale2,
                   float gain, float gain2, float around, int w_one, Join<T> join) {
  constexpr int NM = NS ? NS : MAX_STREAMS;
  const int n = NS ? NS : n_rt;
  extern __shared__ float su[];                      // y, then u of this token
  __shared__ float s_mix[MAX_STREAMS * MAX_STREAMS], s_out[MAX_STREAMS], s_read[MAX_STREAMS], red[32];
  const long long t = blockIdx.x;
  if (y != nullptr) {
    for (int i = threadIdx.x; i < n * n; i += THREADS) s_mix[i] = mix == nullptr ? (i % (n + 1) == 0 ? 1.f : 0.f) : mix[i];
    for (int i = threadIdx.x; i < n; i += THREADS) s_out[i] = out == nullptr ? 1.f : out[i];
  }
  for (int i = threadIdx.x; i < n; i += THREADS) s_read[i] = read == nullptr ? 1.f : read[i];
  __syncthreads();
  float ry = 1.f;
  if (y_weight != nullptr) {
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
      float a[V];
      load_v<V>(y + t * d + i, a);
#pragma unroll
      for (int j = 0; j < V; ++j) ss += a[j] * a[j];
      store_v<V>(su + i, a);                         // this thread reads it back, and puts u there
    }
    ry = 1.f / sqrtf(block_sum(ss, red) / d + y_eps);
  }
  float* Ht = H + t * n * d;
  float sum = 0.f;
  for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
    float x[NM][V], u[V];
#pragma unroll
    for (int s = 0; s < NM; ++s)
      if (NS || s < n) load_v<V>(Ht + static_cast<long long>(s) * d + i, x[s]);
#pragma unroll
    for (int j = 0; j < V; ++j) u[j] = 0.f;
    if (y != nullptr) {
      float b[V];
      if (y_weight != nullptr) {
        float c[V];
        load_v<V>(su + i, b);
        load_v<V>(y_weight + i, c);
#pragma unroll
        for (int j = 0; j < V; ++j) b[j] = b[j] * ry * c[j];
      } else {
        load_v<V>(y + t * d + i, b);
      }
      if (scale != nullptr) {
        float c[V];
        load_v<V>(scale + i, c);
#pragma unroll
        for (int j = 0; j < V; ++j) b[j] *= c[j];
      }
#pragma unroll
      for (int j = 0; j < V; ++j) b[j] *= gain;
      if (y2 != nullptr) {
        float b2[V], c[V];
        load_v<V>(y2 + t * d + i, b2);
        if (scale2 != nullptr) load_v<V>(scale2 + i, c);
#pragma unroll
        for (int j = 0; j < V; ++j) b[j] += gain2 * (scale2 != nullptr ? c[j] * b2[j] : b2[j]);
      }
#pragma unroll(NS ? NS : 1)
      for (int q = 0; q < NM; ++q) {
        if (NS || q < n) {
          float a[V];
#pragma unroll
          for (int j = 0; j < V; ++j) a[j] = s_out[q] * b[j];
#pragma unroll
          for (int s = 0; s < NM; ++s)
            if (NS || s < n) {
              const float m = s_mix[s * n + q];
#pragma unroll
              for (int j = 0; j < V; ++j) a[j] += m * x[s][j];
            }
          if (join.any()) join.template to<V>(a, t, i, d);
          store_v<V>(Ht + static_cast<long long>(q) * d + i, a);
#pragma unroll
          for (int j = 0; j < V; ++j) u[j] += s_read[q] * a[j];
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < NM; ++s)
        if (NS || s < n) {
          if (join.any()) {
            join.template to<V>(x[s], t, i, d);
            store_v<V>(Ht + static_cast<long long>(s) * d + i, x[s]);
          }
#pragma unroll
          for (int j = 0; j < V; ++j) u[j] += s_read[s] * x[s][j];
        }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) sum += rms ? u[j] * u[j] : u[j];
    if (normed != nullptr) store_v<V>(su + i, u);
  }
  if (normed == nullptr) return;                     // a last write with nothing to read after it
  sum = block_sum(sum, red);
  float mean = 0.f, var = sum / d;
  if (!rms) {
    mean = sum / d;
    float dev = 0.f;
    for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
#pragma unroll
      for (int j = 0; j < V; ++j) { const float e = su[i + j] - mean; dev += e * e; }
    }
    var = block_sum(dev, red) / d;
  }
  const float r = 1.f / sqrtf(var + eps);
  for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
    float c[V], o[V];
    load_weight<T, V>(w, w_one, i, c);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = (su[i + j] - mean) * r * (around + c[j]);
    store_v<V>(normed + t * d + i, o);
  }
}

// One plain stream (H += gain scale . y + gain2 scale2 . y2 and what joins, y through its RMS norm where it has a weight, then the norm of H): the whole row in registers,
// NI pieces of V values a thread, every load in flight before the first sum.  TWO: y2 is there.
template <typename T, int V, int NI, bool TWO>
__global__ void __launch_bounds__(THREADS)
residual_step_kernel(float* __restrict__ H, const T* __restrict__ y, const T* __restrict__ y_weight, const T* __restrict__ w, T* __restrict__ normed,
                     int d, float y_eps, float eps, const T* __restrict__ scale, const T* __restrict__ y2, const T* __restrict__ scale2, float gain,
                     float gain2, float around, int w_one, Join<T> join) {
  __shared__ float red[32];
  const long long at = static_cast<long long>(blockIdx.x) * d;
  float x[NI][V], b[NI][V], b2[TWO ? NI : 1][V];
#pragma unroll
  for (int p = 0; p < NI; ++p) {
    const int i = (p * THREADS + threadIdx.x) * V;
#pragma unroll
    for (int j = 0; j < V; ++j) x[p][j] = b[p][j] = 0.f;
    if (i < d) {
      if (y != nullptr) load_v<V>(y + at + i, b[p]);
      if (TWO) load_v<V>(y2 + at + i, b2[p]);
      load_v<V>(H + at + i, x[p]);
    }
  }
  if (y_weight != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int p = 0; p < NI; ++p)
#pragma unroll
      for (int j = 0; j < V; ++j) ss += b[p][j] * b[p][j];
    const float ry = 1.f / sqrtf(block_sum(ss, red) / d + y_eps);
#pragma unroll
    for (int p = 0; p < NI; ++p) {
      const int i = (p * THREADS + threadIdx.x) * V;
      if (i < d) {
        float c[V];
        load_v<V>(y_weight + i, c);
#pragma unroll
        for (int j = 0; j < V; ++j) b[p][j] = b[p][j] * ry * c[j];
      }
    }
  }
  if (scale != nullptr || TWO || gain != 1.f) {
#pragma unroll
    for (int p = 0; p < NI; ++p) {
      const int i = (p * THREADS + threadIdx.x) * V;
      if (i < d) {
        float c[V];
        if (scale != nullptr) {
          load_v<V>(scale + i, c);
#pragma unroll
          for (int j = 0; j < V; ++j) b[p][j] *= c[j];
        }
#pragma unroll
        for (int j = 0; j < V; ++j) b[p][j] *= gain;
        if (TWO) {
          if (scale2 != nullptr) load_v<V>(scale2 + i, c);
#pragma unroll
          for (int j = 0; j < V; ++j) b[p][j] += gain2 * (scale2 != nullptr ? c[j] * b2[p][j] : b2[p][j]);
        }
      }
    }
  }
  if (join.any()) {
#pragma unroll
    for (int p = 0; p < NI; ++p) {
      const int i = (p * THREADS + threadIdx.x) * V;
      if (i < d) join.template to<V>(b[p], blockIdx.x, i, d);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int p = 0; p < NI; ++p) {
    const int i = (p * THREADS + threadIdx.x) * V;
#pragma unroll
    for (int j = 0; j < V; ++j) { x[p][j] += b[p][j]; ss += x[p][j] * x[p][j]; }
    if (i < d) store_v<V>(H + at + i, x[p]);
  }
  if (normed == nullptr) return;
  const float r = 1.f / sqrtf(block_sum(ss, red) / d + eps);
#pragma unroll
  for (int p = 0; p < NI; ++p) {
    const int i = (p * THREADS + threadIdx.x) * V;
    if (i < d) {
      float c[V];
      load_weight<T, V>(w, w_one, i, c);
#pragma unroll
      for (int j = 0; j < V; ++j) c[j] = (around + c[j]) * x[p][j] * r;
      store_v<V>(normed + at + i, c);
    }
  }
}

// x sigmoid(z) times a factor: fp32 models take the exact quotient, bf16 the approximate one (a few parts in 2^22)
template <typename T>
__device__ __forceinline__ float times_sigmoid(float x, float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(x, 1.f + __expf(-z));
  else return x / (1.f + expf(-z));
}

// grid (rows, ceil(F / (THREADS V)))
template <typename T, int V>
__global__ void __launch_bounds__(THREADS)
clamped_glu_kernel(const T* __restrict__ gu, T* __restrict__ out, int F, float limit, float alpha) {
  const long long r = blockIdx.x;
  const int i = (blockIdx.y * THREADS + threadIdx.x) * V;
  if (i >= F) return;
  float g[V], u[V], o[V];
  load_v<V>(gu + r * 2 * F + i, g);
  load_v<V>(gu + r * 2 * F + F + i, u);
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const float a = fminf(g[j], limit), b = fminf(fmaxf(u[j], -limit), limit);
    o[j] = times_sigmoid<T>(a, alpha * a) * (b + 1.f);
  }
  store_v<V>(out + r * F + i, o);
}

// gelu(z) = z sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3)); grid as above
template <typename T, int V>
__global__ void __launch_bounds__(THREADS)
gelu_glu_kernel(const T* __restrict__ gu, T* __restrict__ out, int F) {
  const long long r = blockIdx.x;
  const int i = (blockIdx.y * THREADS + threadIdx.x) * V;
  if (i >= F) return;
  float g[V], u[V];
  load_v<V>(gu + r * 2 * F + i, g);
  load_v<V>(gu + r * 2 * F + F + i, u);
#pragma unroll
  for (int j = 0; j < V; ++j) u[j] *= times_sigmoid<T>(g[j], 1.5957691216057308f * (g[j] + 0.044715f * g[j] * g[j] * g[j]));
  store_v<V>(out + r * F + i, u);
}

template <typename T, int V>
__global__ void __launch_bounds__(THREADS)
sigmoid_gated_norm_kernel(const T* __restrict__ x, const T* __restrict__ gate, const T* __restrict__ w, T* __restrict__ out, int d, float eps) {
  extern __shared__ float sx[];
  __shared__ float red[32];
  const long long t = blockIdx.x;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
    float a[V];
    load_v<V>(x + t * d + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += a[j] * a[j];
    store_v<V>(sx + i, a);
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / d + eps);
  for (int i = threadIdx.x * V; i < d; i += THREADS * V) {
    float g[V], c[V], o[V];
    load_v<V>(gate + t * d + i, g);
    load_v<V>(w + i, c);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = times_sigmoid<T>(sx[i + j] * r * c[j], g[j]);
    store_v<V>(out + t * d + i, o);
  }
}

// grid (rows, ceil(n / (THREADS V)))
template <typename T, int V>
__global__ void __launch_bounds__(THREADS)
softcap_kernel(const T* __restrict__ x, float* __restrict__ out, int n, float cap) {
  const int i = (blockIdx.y * THREADS + threadIdx.x) * V;
  if (i >= n) return;
  const long long at = static_cast<long long>(blockIdx.x) * n + i;
  float a[V];
  load_v<V>(x + at, a);
#pragma unroll
  for (int j = 0; j < V; ++j) a[j] = cap * tanhf(a[j] / cap);
  store_v<V>(out + at, a);
}

template <typename K>
int allow_smem(K kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 220 * 1024) return -3;
  return static_cast<int>(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
}

template <typename T>
int step(float* H, const T* y, const T* y_weight, const T* scale, const float* mix, const float* out, const float* read, const T* w, T* normed,
         long long rows, int n, int d, float y_eps, float eps, int rms, const T* y2, const T* scale2, float gain, float gain2, float around, int w_one,
         const Join<T>& join, cudaStream_t stream) {
  const bool vec = aligned(join.add, 4 * sizeof(T)) && aligned(join.table, 4 * sizeof(T)) && aligned(y2, 4 * sizeof(T)) && aligned(scale2, 4 * sizeof(T)) && d % 4 == 0 && aligned(H, 16) && aligned(y, 4 * sizeof(T)) && aligned(y_weight, 4 * sizeof(T)) && aligned(scale, 4 * sizeof(T)) && (w_one || aligned(w, 4 * sizeof(T))) &&
                   aligned(normed, 4 * sizeof(T));
  if (vec && n == 1 && rms && (y != nullptr || join.any()) && mix == nullptr && out == nullptr && read == nullptr && d <= 32 * THREADS) {
    const int pieces = (d + THREADS * 4 - 1) / (THREADS * 4);
#define DEWB_RES_T(NN, TT) residual_step_kernel<T, 4, NN, TT><<<static_cast<unsigned>(rows), THREADS, 0, stream>>>(H, y, y_weight, w, normed, d, y_eps, eps, \
    scale, y2, scale2, gain, gain2, around, w_one, join)
#define DEWB_RES(NN) do { if (y2 != nullptr) DEWB_RES_T(NN, true); else DEWB_RES_T(NN, false); } while (0)
    if (pieces <= 1) DEWB_RES(1); else if (pieces <= 2) DEWB_RES(2); else if (pieces <= 4) DEWB_RES(4); else DEWB_RES(8);
#undef DEWB_RES
#undef DEWB_RES_T
    return static_cast<int>(cudaGetLastError());
  }
  const size_t smem = static_cast<size_t>(d) * 4;
#define DEWB_STEP(VV, NN) do { const int r = allow_smem(stream_step_kernel<T, VV, NN>, smem); if (r) return r; \
    stream_step_kernel<T, VV, NN><<<static_cast<unsigned>(rows), THREADS, smem, stream>>>(H, y, y_weight, scale, mix, out, read, w, normed, n, d, y_eps, eps, rms, y2, scale2, gain, gain2, around, w_one, join); } while (0)
  if (vec) {
    if (n == 1) DEWB_STEP(4, 1); else if (n == 2) DEWB_STEP(4, 2); else if (n == 3) DEWB_STEP(4, 3); else if (n == 4) DEWB_STEP(4, 4); else DEWB_STEP(1, 0);
  } else {
    DEWB_STEP(1, 0);
  }
#undef DEWB_STEP
  return static_cast<int>(cudaGetLastError());
}

}  // namespace streams
}  // namespace dewb

using namespace dewb::streams;

// `fp32`: activations and weights are fp32, else bf16.  `positions` / `pos` may be null.
extern "C" int dewb_embed_streams(const long long* tokens, const int* positions, const void* embed, const void* pos, float* H, long long rows,
                                  int n, int d, int vocab, int max_pos, float gain, int fp32, void* stream_ptr) {
  if (rows <= 0) return 0;
  if (n < 1 || d < 1 || vocab < 1 || (pos != nullptr && (max_pos < 1 || positions == nullptr))) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bool vec = d % 4 == 0 && aligned(H, 16) && aligned(embed, 16) && aligned(pos, 16);
  const unsigned grid = static_cast<unsigned>(rows);
#define DEWB_EMBED(TT, VV) embed_streams_kernel<TT, VV><<<grid, THREADS, 0, stream>>>(tokens, positions, static_cast<const TT*>(embed), \
    static_cast<const TT*>(pos), H, n, d, vocab, max_pos > 0 ? max_pos : 1, gain)
  if (fp32) { if (vec) DEWB_EMBED(float, 4); else DEWB_EMBED(float, 1); }
  else { if (vec) DEWB_EMBED(bf16, 4); else DEWB_EMBED(bf16, 1); }
#undef DEWB_EMBED
  return static_cast<int>(cudaGetLastError());
}

// H [rows, n, d] fp32, updated in place when `y` [rows, d] is given; normed [rows, d] (null: write only).  mix is indexed [from, to].  `mix`, `out`
// and `read` may be null (each stream keeps itself, takes y, and is read with weight 1); y_weight [d]: y passes an RMS norm with that weight first.
// `scale`, `scale2` [d], y2 [rows, d]: see stream_step above (null: absent); weights of the norm are `around` + w, w [d] or (`w_one`) one number.  `add` [d]
// and `table_gain` times `table` [vocab, d] at the row's token join the one stream (n 1) as well (null: neither).
extern "C" int dewb_stream_step(float* H, const void* y, const void* y_weight, const void* scale, const float* mix, const float* out,
                                const float* read, const void* w, void* normed, long long rows, int n, int d, float y_eps, float eps, int rms,
                                const void* y2, const void* scale2, float gain, float gain2, float around, int w_one, const void* add, const void* table,
                                const long long* tokens, int vocab, float table_gain, int fp32, void* stream_ptr) {
  if (rows <= 0) return 0;
  if (n < 1 || n > MAX_STREAMS || d < 1 || (y == nullptr && (y_weight != nullptr || y2 != nullptr)) || (y_weight != nullptr && y2 != nullptr) || (normed != nullptr && w == nullptr) ||
      ((add != nullptr || table != nullptr) && n != 1) || (table != nullptr && (tokens == nullptr || vocab < 1)))
    return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (fp32) return step<float>(H, static_cast<const float*>(y), static_cast<const float*>(y_weight), static_cast<const float*>(scale), mix, out, read,
                               static_cast<const float*>(w), static_cast<float*>(normed), rows, n, d, y_eps, eps, rms, static_cast<const float*>(y2),
                               static_cast<const float*>(scale2), gain, gain2, around, w_one,
                               Join<float>{static_cast<const float*>(add), static_cast<const float*>(table), tokens, vocab, table_gain}, stream);
  return step<bf16>(H, static_cast<const bf16*>(y), static_cast<const bf16*>(y_weight), static_cast<const bf16*>(scale), mix, out, read,
                    static_cast<const bf16*>(w), static_cast<bf16*>(normed), rows, n, d, y_eps, eps, rms, static_cast<const bf16*>(y2),
                    static_cast<const bf16*>(scale2), gain, gain2, around, w_one,
                    Join<bf16>{static_cast<const bf16*>(add), static_cast<const bf16*>(table), tokens, vocab, table_gain}, stream);
}

// x [rows, n] -> out [rows, n] fp32
extern "C" int dewb_softcap(const void* x, float* out, long long rows, int n, float cap, int fp32, void* stream_ptr) {
  if (rows <= 0) return 0;
  if (n < 1 || !(cap > 0.f)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const int v = n % 4 == 0 && aligned(x, 16) && aligned(out, 16) ? 4 : 1;
  const int blocks = (n + THREADS * v - 1) / (THREADS * v);
  if (blocks > 65535) return -3;
  const dim3 grid(static_cast<unsigned>(rows), blocks);
#define DEWB_CAP(TT, VV) softcap_kernel<TT, VV><<<grid, THREADS, 0, stream>>>(static_cast<const TT*>(x), out, n, cap)
  if (fp32) { if (v == 4) DEWB_CAP(float, 4); else DEWB_CAP(float, 1); }
  else { if (v == 4) DEWB_CAP(bf16, 4); else DEWB_CAP(bf16, 1); }
#undef DEWB_CAP
  return static_cast<int>(cudaGetLastError());
}

// gu [rows, 2 F] (gate half, then linear half) -> out [rows, F]
extern "C" int dewb_clamped_glu(const void* gu, void* out, long long rows, int F, float limit, float alpha, int fp32, void* stream_ptr) {
  if (rows <= 0) return 0;
  if (F < 1) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const int v = F % 8 == 0 && !fp32 && aligned(gu, 16) && aligned(out, 16) ? 8 : F % 4 == 0 && aligned(gu, 16) && aligned(out, 16) ? 4 : 1;
  const int blocks = (F + THREADS * v - 1) / (THREADS * v);
  if (blocks > 65535) return -3;
  const dim3 grid(static_cast<unsigned>(rows), blocks);
#define DEWB_GLU(TT, VV) clamped_glu_kernel<TT, VV><<<grid, THREADS, 0, stream>>>(static_cast<const TT*>(gu), static_cast<TT*>(out), F, limit, alpha)
  if (fp32) { if (v == 4) DEWB_GLU(float, 4); else DEWB_GLU(float, 1); }
  else { if (v == 8) DEWB_GLU(bf16, 8); else if (v == 4) DEWB_GLU(bf16, 4); else DEWB_GLU(bf16, 1); }
#undef DEWB_GLU
  return static_cast<int>(cudaGetLastError());
}

// gu [rows, 2 F] (gate half, then linear half) -> out [rows, F]
extern "C" int dewb_gelu_glu(const void* gu, void* out, long long rows, int F, int fp32, void* stream_ptr) {
  if (rows <= 0) return 0;
  if (F < 1) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bool a16 = aligned(gu, 16) && aligned(out, 16);
  const int v = F % 8 == 0 && !fp32 && a16 ? 8 : F % 4 == 0 && a16 ? 4 : 1;
  const int blocks = (F + THREADS * v - 1) / (THREADS * v);
  if (blocks > 65535) return -3;
  const dim3 grid(static_cast<unsigned>(rows), blocks);
#define DEWB_GELU(TT, VV) gelu_glu_kernel<TT, VV><<<grid, THREADS, 0, stream>>>(static_cast<const TT*>(gu), static_cast<TT*>(out), F)
  if (fp32) { if (v == 4) DEWB_GELU(float, 4); else DEWB_GELU(float, 1); }
  else { if (v == 8) DEWB_GELU(bf16, 8); else if (v == 4) DEWB_GELU(bf16, 4); else DEWB_GELU(bf16, 1); }
#undef DEWB_GELU
  return static_cast<int>(cudaGetLastError());
}

extern "C" int dewb_sigmoid_gated_norm(const void* x, const void* gate, const void* w, void* out, long long rows, int d, float eps, int fp32,
                                       void* stream_ptr) {
  if (rows <= 0) return 0;
  if (d < 1) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const bool vec = d % 4 == 0 && aligned(x, 16) && aligned(gate, 16) && aligned(w, 16) && aligned(out, 16);
  const size_t smem = static_cast<size_t>(d) * 4;
  const unsigned grid = static_cast<unsigned>(rows);
#define DEWB_GN(TT, VV) do { const int r = allow_smem(sigmoid_gated_norm_kernel<TT, VV>, smem); if (r) return r; \
    sigmoid_gated_norm_kernel<TT, VV><<<grid, THREADS, smem, stream>>>(static_cast<const TT*>(x), static_cast<const TT*>(gate), \
        static_cast<const TT*>(w), static_cast<TT*>(out), d, eps); } while (0)
  if (fp32) { if (vec) DEWB_GN(float, 4); else DEWB_GN(float, 1); }
  else { if (vec && d % 8 == 0) DEWB_GN(bf16, 8); else if (vec) DEWB_GN(bf16, 4); else DEWB_GN(bf16, 1); }
#undef DEWB_GN
  return static_cast<int>(cudaGetLastError());
}
