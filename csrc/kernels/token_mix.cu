// What a token takes from its neighbours, and the small products and norms around a recurrence, for sm_100a.
//
//   conv_tokens     a short causal convolution per channel over a call's tokens, behind the bias of the projection it follows, with or without silu;
//                   the inputs in front of the call's first token come from the row's state, zeros at a sequence's start
//   conv_tail       the row's state after the call: its last taps - 1 inputs (taps 2: the previous token itself)
//   conv_step       both for one token per row
//   shift_tokens    n mixes of every token with the one before it, x + (x' - x) mu_j
//   narrow_product  x w^T with few outputs, kept in fp32 (gates of a recurrence)
//   low_rank_decay  -exp(w2 tanh(z) + w0): the logarithm of a decay per channel through a bottleneck
//   head_gated_norm RMS norm of every head, times a weight (one head's, or all heads'), times silu or sigmoid of a gate
//
// Rows of a call may lie anywhere in the store (`row_ids`); positions below 0 are padding at a row's end: they leave no trace and give zeros.
// Activations are bf16 or fp32 (template T), states and sums fp32.  Compiled without fast math.
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/mma_bf16.cuh"
#include "../common/rows.cuh"

namespace dewb {
namespace tokenmix {

using namespace rows;

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

constexpr int RUN = 16;          // tokens a thread walks
constexpr int MAX_TAPS = 64;

// x [R, S, row_stride] -> y [R, S, C]; state [store rows, C, taps - 1] (null: nothing before the call).  grid (channel blocks, token runs, R).
// TAPS 0: any number of taps, re-read from memory; else the inputs slide through registers.
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(128)
conv_tokens_kernel(const T* __restrict__ x, long long row_stride, const T* __restrict__ bias, const T* __restrict__ w, const float* __restrict__ state,
                   const int* __restrict__ positions, const int* __restrict__ row_ids, int S, int C, int taps_rt, int act, T* __restrict__ y) {
  const int taps = TAPS ? TAPS : taps_rt;
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, row = blockIdx.z, t0 = blockIdx.y * RUN;
  if (c >= C) return;
  const int* pos = positions + static_cast<long long>(row) * S;
  const T* xr = x + static_cast<long long>(row) * S * row_stride + c;
  T* yr = y + static_cast<long long>(row) * S * C + c;
  const int r = row_ids == nullptr ? row : row_ids[row];
  const float* st_row = state != nullptr && pos[0] > 0 ? state + (static_cast<long long>(r) * C + c) * (taps - 1) : nullptr;
  float b[V];
#pragma unroll
  for (int j = 0; j < V; ++j) b[j] = 0.f;
  if (bias != nullptr) load_v<V>(bias + c, b);
  auto input = [&](int t, float (&u)[V]) {
    if (t >= 0) {
      load_v<V>(xr + t * row_stride, u);
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] += b[j];
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] = st_row != nullptr ? st_row[j * (taps - 1) + taps - 1 + t] : 0.f;
    }
  };
  auto finish = [&](int t, float (&o)[V]) {
    if (act) {
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] = sizeof(T) == 2 ? __fdividef(o[j], 1.f + __expf(-o[j])) : o[j] * sigmoid(o[j]);
    }
    store_v<V>(yr + static_cast<long long>(t) * C, o);
  };
  const int t1 = min(S, t0 + RUN);
  if constexpr (TAPS > 0) {
    constexpr int AHEAD = 4;                      // tokens fetched together
    float wt[V][TAPS], u[TAPS + AHEAD - 1][V];
#pragma unroll
    for (int j = 0; j < V; ++j)
#pragma unroll
      for (int q = 0; q < TAPS; ++q) wt[j][q] = ld(w + static_cast<long long>(c + j) * TAPS + q);
#pragma unroll
    for (int q = 0; q + 1 < TAPS; ++q) input(t0 - TAPS + 1 + q, u[AHEAD + q]);
    for (int t = t0; t < t1; t += AHEAD) {
#pragma unroll
      for (int q = 0; q + 1 < TAPS; ++q)
#pragma unroll
        for (int j = 0; j < V; ++j) u[q][j] = u[q + AHEAD][j];
#pragma unroll
      for (int s = 0; s < AHEAD; ++s)
        if (t + s < t1) input(t + s, u[TAPS - 1 + s]);
#pragma unroll
      for (int s = 0; s < AHEAD; ++s) {
        if (t + s >= t1) break;
        float o[V];
        const bool live = pos[t + s] >= 0;
#pragma unroll
        for (int j = 0; j < V; ++j) {
          o[j] = 0.f;
#pragma unroll
          for (int q = 0; q < TAPS; ++q) o[j] += wt[j][q] * u[q + s][j];
          if (!live) o[j] = 0.f;
        }
        finish(t + s, o);
      }
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float o[V];
#pragma unroll
      for (int j = 0; j < V; ++j) o[j] = 0.f;
      if (pos[t] >= 0) {
        for (int q = 0; q < taps; ++q) {
          float u[V];
          input(t - taps + 1 + q, u);
#pragma unroll
          for (int j = 0; j < V; ++j) o[j] += ld(w + static_cast<long long>(c + j) * taps + q) * u[j];
        }
      }
      finish(t, o);
    }
  }
}

// state [store rows, C, keep] after a call: the last `keep` inputs of the row.  A thread owns a channel of a row; place j takes what stood further on
// (or an input of the call), so the walk upwards reads every place before it is overwritten.
template <typename T>
__global__ void __launch_bounds__(128)
conv_tail_kernel(const T* __restrict__ x, long long row_stride, const T* __restrict__ bias, const int* __restrict__ positions,
                 const int* __restrict__ lengths, const int* __restrict__ row_ids, int S, int C, int keep, float* __restrict__ state) {
  const int c = blockIdx.x * 128 + threadIdx.x, row = blockIdx.y;
  const int first = positions[static_cast<long long>(row) * S];
  if (c >= C || first < 0) return;
  const int n = min(lengths[row] - first, S);
  float* s = state + (static_cast<long long>(row_ids == nullptr ? row : row_ids[row]) * C + c) * keep;
  const float b = bias == nullptr ? 0.f : ld(bias + c);
  for (int j = 0; j < keep; ++j) {
    const int t = n - keep + j;
    s[j] = t >= 0 ? ld(x + (static_cast<long long>(row) * S + t) * row_stride + c) + b : first > 0 ? s[keep + t] : 0.f;
  }
}

// One token per row: y [R, C], and the state moves on.
template <typename T>
__global__ void __launch_bounds__(128)
conv_step_kernel(const T* __restrict__ x, long long row_stride, const T* __restrict__ bias, const T* __restrict__ w, float* __restrict__ state,
                 const int* __restrict__ positions, const int* __restrict__ row_ids, int C, int taps, int act, T* __restrict__ y) {
  const int c = blockIdx.x * 128 + threadIdx.x, row = blockIdx.y;
  if (c >= C) return;
  const int p = positions[row], keep = taps - 1;
  T* out = y + static_cast<long long>(row) * C + c;
  if (p < 0) { st(out, 0.f); return; }
  const float u = ld(x + row * row_stride + c) + (bias == nullptr ? 0.f : ld(bias + c));
  const T* wc = w + static_cast<long long>(c) * taps;
  float* s = state + (static_cast<long long>(row_ids == nullptr ? row : row_ids[row]) * C + c) * keep;
  float o = ld(wc + keep) * u;
  for (int j = 0; j < keep; ++j) {
    const float v = p > 0 ? s[j] : 0.f;
    o += ld(wc + j) * v;
    if (j > 0) s[j - 1] = v;
  }
  if (keep > 0) s[keep - 1] = u;
  st(out, act ? o * sigmoid(o) : o);
}

// x [R, S, d], mu [n, d] -> out [n, R * S, d]; state [store rows, d] holds the token before the call's first (written here when S is 1).
template <typename T, int V>
__global__ void __launch_bounds__(128)
shift_tokens_kernel(const T* __restrict__ x, const T* __restrict__ mu, float* __restrict__ state, const int* __restrict__ positions,
                    const int* __restrict__ row_ids, int S, int d, int n, long long tokens, T* __restrict__ out) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * V;
  if (c >= d) return;
  const long long t = blockIdx.x, row = t / S;
  const int first = positions[row * S];
  const bool live = positions[t] >= 0;
  float a[V], before[V];
#pragma unroll
  for (int j = 0; j < V; ++j) before[j] = 0.f;
  load_v<V>(x + t * d + c, a);
  float* s = state == nullptr ? nullptr : state + static_cast<long long>(row_ids == nullptr ? row : row_ids[row]) * d + c;
  if (t > row * S) load_v<V>(x + (t - 1) * d + c, before);
  else if (s != nullptr && first > 0) load_v<V>(s, before);
  for (int i = 0; i < n; ++i) {
    float m[V], o[V];
    load_v<V>(mu + static_cast<long long>(i) * d + c, m);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = live ? a[j] + (before[j] - a[j]) * m[j] : 0.f;
    store_v<V>(out + (i * tokens + t) * d + c, o);
  }
  if (S == 1 && live && s != nullptr) store_v<V>(s, a);
}

// out [T, n] fp32 = x [T, d] w [n, d]^T.  A block forms NOUT outputs of NTOK tokens; its warps share the reduction.  grid (ceil(n / NOUT), ceil(T / NTOK)).
constexpr int NTOK = 4, NOUT = 4;
template <typename T, int V>
__global__ void __launch_bounds__(256)
narrow_product_kernel(const T* __restrict__ x, const T* __restrict__ w, float* __restrict__ out, long long tokens, int n, int d) {
  __shared__ float part[8][NTOK * NOUT];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, e0 = blockIdx.x * NOUT;
  const long long t0 = static_cast<long long>(blockIdx.y) * NTOK;
  float acc[NTOK][NOUT] = {};
  for (int c = threadIdx.x * V; c < d; c += 256 * V) {
    float a[NTOK][V], b[NOUT][V];
#pragma unroll
    for (int i = 0; i < NTOK; ++i) load_v<V>(x + min(t0 + i, tokens - 1) * d + c, a[i]);
#pragma unroll
    for (int e = 0; e < NOUT; ++e) load_v<V>(w + static_cast<long long>(min(e0 + e, n - 1)) * d + c, b[e]);
#pragma unroll
    for (int i = 0; i < NTOK; ++i)
#pragma unroll
      for (int e = 0; e < NOUT; ++e)
#pragma unroll
        for (int j = 0; j < V; ++j) acc[i][e] += a[i][j] * b[e][j];
  }
#pragma unroll
  for (int i = 0; i < NTOK; ++i)
#pragma unroll
    for (int e = 0; e < NOUT; ++e) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) acc[i][e] += __shfl_xor_sync(0xffffffffu, acc[i][e], o);
      if (lane == 0) part[warp][i * NOUT + e] = acc[i][e];
    }
  __syncthreads();
  if (threadIdx.x < NTOK * NOUT) {
    const int i = threadIdx.x / NOUT, e = e0 + threadIdx.x % NOUT;
    float s = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) s += part[q][threadIdx.x];
    if (t0 + i < tokens && e < n) out[(t0 + i) * n + e] = s;
  }
}

// z [T, ld] fp32, w2 [C, rank], w0 [C] -> out [T, C] = -exp(w2 tanh(z) + w0).  fp32 form: a thread per channel, 8 tokens.
template <typename T>
__global__ void __launch_bounds__(128)
low_rank_decay_kernel(const float* __restrict__ z, long long ldz, const T* __restrict__ w2, const T* __restrict__ w0, float* __restrict__ out,
                      long long tokens, int C, int rank) {
  extern __shared__ float sz[];                       // [8][rank]
  const long long t0 = static_cast<long long>(blockIdx.x) * 8;
  for (int i = threadIdx.x; i < 8 * rank; i += 128) {
    const int t = i / rank, k = i - t * rank;
    sz[i] = t0 + t < tokens ? tanhf(z[(t0 + t) * ldz + k]) : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c >= C) return;
  float acc[8] = {};
  for (int k = 0; k < rank; ++k) {
    const float b = ld(w2 + static_cast<long long>(c) * rank + k);
#pragma unroll
    for (int t = 0; t < 8; ++t) acc[t] += sz[t * rank + k] * b;
  }
  const float bias = ld(w0 + c);
#pragma unroll
  for (int t = 0; t < 8; ++t) if (t0 + t < tokens) out[(t0 + t) * C + c] = -expf(acc[t] + bias);
}

// The same on the tensor cores: a warp forms 16 tokens x 64 channels; tanh(z) goes in as two bf16 numbers, so nothing of it is lost that matters in fp32.
__global__ void __launch_bounds__(128)
low_rank_decay_mma_kernel(const float* __restrict__ z, long long ldz, const bf16* __restrict__ w2, const bf16* __restrict__ w0, float* __restrict__ out,
                          long long tokens, int C, int rank) {
  using namespace mma16;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t2 = (lane & 3) * 2;
  const long long t0 = static_cast<long long>(blockIdx.x) * 16;
  const int c0 = (blockIdx.y * 4 + warp) * 64;
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  for (int k0 = 0; k0 < rank; k0 += 16) {
    uint32_t big[4], rest[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const long long t = t0 + g + 8 * (x & 1);
      const int k = k0 + t2 + 8 * (x >> 1);
      const float a = t < tokens && k < rank ? tanhf(z[t * ldz + k]) : 0.f, b = t < tokens && k + 1 < rank ? tanhf(z[t * ldz + k + 1]) : 0.f;
      split2(a, b, big[x], rest[x]);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = c0 + j * 8 + g;
      uint32_t b[2] = {0u, 0u};
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int k = k0 + t2 + 8 * x;                // rank is even: a pair lies in the row or past it
        if (c < C && k < rank) b[x] = *reinterpret_cast<const uint32_t*>(w2 + static_cast<long long>(c) * rank + k);
      }
      mma(acc[j], big, b[0], b[1]);
      mma(acc[j], rest, b[0], b[1]);
    }
  }
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const long long t = t0 + g + 8 * (e >> 1);
      const int c = c0 + j * 8 + t2 + (e & 1);
      if (t < tokens && c < C) out[t * C + c] = -expf(acc[j][e] + __bfloat162float(w0[c]));
    }
}

// x [T, H, d], gate [T, *] (head h's columns start at h d), w [d] or [H d] -> out [T, H d].  LG lanes per (token, head).
template <typename T, int V, int LG>
__global__ void __launch_bounds__(256)
head_gated_norm_kernel(const T* __restrict__ x, const T* __restrict__ gate, long long gate_stride, const T* __restrict__ w, int shared_w, float eps,
                       int silu, long long items, int H, int d, T* __restrict__ out) {
  const long long item = static_cast<long long>(blockIdx.x) * (256 / LG) + threadIdx.x / LG;
  const int lane = threadIdx.x % LG;
  const bool on = item < items;                       // every lane stays for the sums
  const long long t = on ? item / H : 0;
  const int h = on ? static_cast<int>(item - t * H) : 0;
  const T* src = x + (on ? item : 0) * d;
  float ss = 0.f;
  for (int i = lane * V; i < d; i += LG * V) {
    float a[V];
    load_v<V>(src + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += a[j] * a[j];
  }
#pragma unroll
  for (int o = LG / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!on) return;
  const float r = 1.f / sqrtf(ss / d + eps);
  for (int i = lane * V; i < d; i += LG * V) {
    float a[V], z[V], c[V];
    load_v<V>(src + i, a);
    load_v<V>(gate + t * gate_stride + h * d + i, z);
    load_v<V>(w + (shared_w ? 0 : h * d) + i, c);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float s = sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-z[j])) : sigmoid(z[j]);
      a[j] = a[j] * r * c[j] * (silu ? z[j] * s : s);
    }
    store_v<V>(out + item * d + i, a);
  }
}

template <typename T>
int conv_any(const T* x, long long rs, const T* bias, const T* w, float* state, const int* positions, const int* lengths, const int* row_ids, int R, int S,
             int C, int taps, int act, T* y, cudaStream_t stream) {
  if (S == 1 && state != nullptr) {
    conv_step_kernel<T><<<dim3((C + 127) / 128, R), 128, 0, stream>>>(x, rs, bias, w, state, positions, row_ids, C, taps, act, y);
    return static_cast<int>(cudaGetLastError());
  }
  constexpr int W = sizeof(T) == 2 ? 8 : 4;
  const bool vec = C % W == 0 && rs % W == 0 && aligned(x, 16) && aligned(bias, 16) && aligned(y, 16);
  const int per = 128 * (vec ? W : 1);
  const dim3 grid((C + per - 1) / per, (S + RUN - 1) / RUN, R);
  if (grid.y > 65535u) return -3;
#define DEWB_CONV(VV, KK) conv_tokens_kernel<T, VV, KK><<<grid, 128, 0, stream>>>(x, rs, bias, w, state, positions, row_ids, S, C, taps, act, y)
  if (vec) { if (taps == 4) DEWB_CONV(W, 4); else if (taps == 3) DEWB_CONV(W, 3); else if (taps == 2) DEWB_CONV(W, 2); else DEWB_CONV(W, 0); }
  else DEWB_CONV(1, 0);
#undef DEWB_CONV
  if (state != nullptr && taps > 1)
    conv_tail_kernel<T><<<dim3((C + 127) / 128, R), 128, 0, stream>>>(x, rs, bias, positions, lengths, row_ids, S, C, taps - 1, state);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int shift_any(const T* x, const T* mu, float* state, const int* positions, const int* lengths, const int* row_ids, int R, int S, int d, int n, T* out,
              cudaStream_t stream) {
  constexpr int W = sizeof(T) == 2 ? 8 : 4;
  const bool vec = d % W == 0 && aligned(x, 16) && aligned(mu, 16) && aligned(out, 16) && aligned(state, 16);
  const int per = 128 * (vec ? W : 1);
  const long long tokens = static_cast<long long>(R) * S;
  const dim3 grid(static_cast<unsigned>(tokens), (d + per - 1) / per);
  if (vec) shift_tokens_kernel<T, W><<<grid, 128, 0, stream>>>(x, mu, state, positions, row_ids, S, d, n, tokens, out);
  else shift_tokens_kernel<T, 1><<<grid, 128, 0, stream>>>(x, mu, state, positions, row_ids, S, d, n, tokens, out);
  if (state != nullptr && S > 1) conv_tail_kernel<T><<<dim3((d + 127) / 128, R), 128, 0, stream>>>(x, d, nullptr, positions, lengths, row_ids, S, d, 1, state);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace tokenmix
}  // namespace dewb

using namespace dewb::tokenmix;

// x [R * S, row_stride >= C] -> y [R, S, C]; bias [C] (null: none), w [C, taps], state [store rows, C, taps - 1] (null: nothing before, nothing kept);
// lengths [R]: the position after a row's last token.  `act`: silu.
extern "C" int dewb_conv_tokens(const void* x, long long row_stride, const void* bias, const void* w, float* state, const int* positions, const int* lengths,
                                const int* row_ids, int R, int S, int C, int taps, int act, void* y, int fp32, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (C < 1 || taps < 1 || taps > MAX_TAPS || row_stride < C || R > 65535 || (state != nullptr && lengths == nullptr)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (fp32) return conv_any<float>(static_cast<const float*>(x), row_stride, static_cast<const float*>(bias), static_cast<const float*>(w), state, positions,
                                   lengths, row_ids, R, S, C, taps, act, static_cast<float*>(y), stream);
  return conv_any<dewb::rows::bf16>(static_cast<const dewb::rows::bf16*>(x), row_stride, static_cast<const dewb::rows::bf16*>(bias),
                                    static_cast<const dewb::rows::bf16*>(w), state, positions, lengths, row_ids, R, S, C, taps, act,
                                    static_cast<dewb::rows::bf16*>(y), stream);
}

// x [R, S, d], mu [n, d] -> out [n, R, S, d]; state [store rows, d] (null: zeros before every row, nothing kept)
extern "C" int dewb_shift_tokens(const void* x, const void* mu, float* state, const int* positions, const int* lengths, const int* row_ids, int R, int S, int d,
                                 int n, void* out, int fp32, void* stream_ptr) {
  if (R <= 0 || S <= 0) return 0;
  if (d < 1 || n < 1 || R > 65535 || (state != nullptr && lengths == nullptr)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (fp32) return shift_any<float>(static_cast<const float*>(x), static_cast<const float*>(mu), state, positions, lengths, row_ids, R, S, d, n,
                                    static_cast<float*>(out), stream);
  return shift_any<dewb::rows::bf16>(static_cast<const dewb::rows::bf16*>(x), static_cast<const dewb::rows::bf16*>(mu), state, positions, lengths, row_ids, R, S, d,
                                     n, static_cast<dewb::rows::bf16*>(out), stream);
}

// out [tokens, n] fp32 = x [tokens, d] w [n, d]^T
extern "C" int dewb_narrow_product(const void* x, const void* w, float* out, long long tokens, int n, int d, int fp32, void* stream_ptr) {
  if (tokens <= 0) return 0;
  const long long groups = (tokens + NTOK - 1) / NTOK;
  if (n < 1 || d < 1 || groups > 65535) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const dim3 grid((n + NOUT - 1) / NOUT, static_cast<unsigned>(groups));
  const bool a16 = aligned(x, 16) && aligned(w, 16);
#define DEWB_NARROW(TT, VV) narrow_product_kernel<TT, VV><<<grid, 256, 0, stream>>>(static_cast<const TT*>(x), static_cast<const TT*>(w), out, tokens, n, d)
  if (fp32) { if (a16 && d % 4 == 0) DEWB_NARROW(float, 4); else DEWB_NARROW(float, 1); }
  else { if (a16 && d % 8 == 0) DEWB_NARROW(bf16, 8); else DEWB_NARROW(bf16, 1); }
#undef DEWB_NARROW
  return static_cast<int>(cudaGetLastError());
}

// z [tokens, ldz] fp32, w2 [C, rank], w0 [C] -> out [tokens, C] fp32
extern "C" int dewb_low_rank_decay(const float* z, long long ldz, const void* w2, const void* w0, float* out, long long tokens, int C, int rank, int fp32,
                                   void* stream_ptr) {
  if (tokens <= 0) return 0;
  if (C < 1 || rank < 1 || rank > 1024 || ldz < rank || (C + 127) / 128 > 65535) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  if (!fp32 && rank % 2 == 0 && aligned(w2, 4)) {
    low_rank_decay_mma_kernel<<<dim3(static_cast<unsigned>((tokens + 15) / 16), (C + 255) / 256), 128, 0, stream>>>(z, ldz, static_cast<const bf16*>(w2),
                                                                                                               static_cast<const bf16*>(w0), out, tokens, C, rank);
    return static_cast<int>(cudaGetLastError());
  }
  const dim3 grid(static_cast<unsigned>((tokens + 7) / 8), (C + 127) / 128);
  const size_t smem = static_cast<size_t>(8) * rank * 4;
  if (fp32) low_rank_decay_kernel<float><<<grid, 128, smem, stream>>>(z, ldz, static_cast<const float*>(w2), static_cast<const float*>(w0), out, tokens, C, rank);
  else low_rank_decay_kernel<bf16><<<grid, 128, smem, stream>>>(z, ldz, static_cast<const bf16*>(w2), static_cast<const bf16*>(w0), out, tokens, C, rank);
  return static_cast<int>(cudaGetLastError());
}

// x [tokens, H, d], gate [tokens, gate_stride], w [d] (`shared_w`) or [H d] -> out [tokens, H d]
extern "C" int dewb_head_gated_norm(const void* x, const void* gate, long long gate_stride, const void* w, int shared_w, float eps, int silu, long long tokens,
                                    int H, int d, void* out, int fp32, void* stream_ptr) {
  if (tokens <= 0) return 0;
  if (H < 1 || d < 1 || gate_stride < static_cast<long long>(H) * d) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const long long items = tokens * H;
  const bool a16 = aligned(x, 16) && aligned(gate, 16) && aligned(w, 16) && aligned(out, 16);
  const int v = a16 && !fp32 && d % 8 == 0 && gate_stride % 8 == 0 ? 8 : a16 && d % 4 == 0 && gate_stride % 4 == 0 ? 4 : 1;
  const int lg = d <= 8 * v ? 8 : d <= 16 * v ? 16 : 32;
  const long long blocks = (items * lg + 255) / 256;
  if (blocks > 0x7fffffffll) return -3;
#define DEWB_HGN(TT, VV, LL) head_gated_norm_kernel<TT, VV, LL><<<static_cast<unsigned>(blocks), 256, 0, stream>>>(static_cast<const TT*>(x), \
    static_cast<const TT*>(gate), gate_stride, static_cast<const TT*>(w), shared_w, eps, silu, items, H, d, static_cast<TT*>(out))
#define DEWB_HGN_L(TT, VV) do { if (lg == 8) DEWB_HGN(TT, VV, 8); else if (lg == 16) DEWB_HGN(TT, VV, 16); else DEWB_HGN(TT, VV, 32); } while (0)
  if (fp32) { if (v == 4) DEWB_HGN_L(float, 4); else DEWB_HGN_L(float, 1); }
  else { if (v == 8) DEWB_HGN_L(bf16, 8); else if (v == 4) DEWB_HGN_L(bf16, 4); else DEWB_HGN_L(bf16, 1); }
#undef DEWB_HGN_L
#undef DEWB_HGN
  return static_cast<int>(cudaGetLastError());
}
