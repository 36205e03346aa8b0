// Recurrences over a matrix state per head whose decays come from the token, for sm_100a.  k and q have dk entries, v has dv, S is [dk, dv] in fp32.
//
//   delta    k^ = k / sqrt(|k|^2 + 1e-6), q^ likewise times `scale`; a step beta = sigmoid(zb) and a decay g = exp(-e^A_log softplus(za + dt_bias)) per head:
//            S' = g S + k^ (x) beta (v - g k^ S),   o = q^ S'.   A group of heads may share q and k.
//   memory   log gates per head, soft-capped: i = cap tanh((zi + bi) / cap) and f = log sigmoid(cap tanh((zf + bf) / cap)).  With M' = max(f + M, i), M = 0 at
//            first, the old state keeps e^(f + M - M') and k (x) v enters with e^(i - M'); the normaliser n goes the same way with k alone;
//            o = scale q S' / (max(|scale q n'|, e^-M') + 1e-6)
//   wkv      a decay w per key channel, given by its logarithm, and a bonus u for the token itself:  o = q S + (sum_c q_c u_c k_c) v,   S' = w . S + k (x) v
//
//   gated_step      one token per row: the state is read and written once
//   gated_sequence  a call's tokens one after another in fp32, any head widths up to 512 (the exact form; it serves fp32 models)
//
// A call row whose first position is 0 starts from zero; positions below 0 are padding at a row's end: they change no state and give zeros.
// q, k and v lie in rows of `row_stride` values; inputs and outputs are bf16 or fp32 (template T), everything else fp32.  Compiled without fast math.
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/gated_rule.cuh"

namespace dewb {
namespace gated {

constexpr int STEP_THREADS = 256;

// grid (H, column tiles, rows); a block walks its column tiles (memory: one block per row and head, which also owns n and m).  A thread owns V columns of
// the key rows group, group + GROUPS, ..., U of them.
template <int MODE, typename T, int V, int LANES, int U>
__global__ void __launch_bounds__(STEP_THREADS, U > 16 ? 1 : U * V > 32 ? 2 : 3)
gated_step_kernel(Args<T> p) {
  constexpr int GROUPS = STEP_THREADS / LANES, TILE = LANES * V;
  extern __shared__ float sm[];                 // q [dk], k [dk], w [dk] (wkv), partial [GROUPS][TILE], u [TILE]
  __shared__ float red[32];
  const int dk = p.dk, dv = p.dv;
  float *sq = sm, *sk = sq + dk, *sw = sk + dk, *part = sw + (MODE == WKV ? dk : 0), *su = part + GROUPS * TILE;
  const int h = blockIdx.x, row = blockIdx.z, pos = p.positions[row];
  const int lane = threadIdx.x % LANES, group = threadIdx.x / LANES;
  T* o = p.out + (static_cast<long long>(row) * p.H + h) * dv;
  if (pos < 0) {
    for (int t0 = blockIdx.y * TILE; t0 < dv; t0 += gridDim.y * TILE)
      for (int c = threadIdx.x; c < TILE; c += STEP_THREADS) if (t0 + c < dv) st(o + t0 + c, 0.f);
    return;
  }
  const bool fresh = pos == 0;
  const int r = p.row_ids == nullptr ? row : p.row_ids[row];
  const long long rh = static_cast<long long>(r) * p.H + h;
  const int g = h / (p.H / p.G);
  const T *q = p.q + row * p.q_stride + g * dk, *k = p.k + row * p.k_stride + g * dk, *v = p.v + row * p.v_stride + h * dv;
  float a = 0.f, b = 0.f, c = 0.f;              // what the mode needs of the token's scalars
  float s0 = 0.f, s1 = 0.f;
  for (int i = threadIdx.x; i < dk; i += STEP_THREADS) {
    const float x = ld(q + i), y = ld(k + i);
    sq[i] = x;
    sk[i] = y;
    if (MODE == DELTA) { s0 += x * x; s1 += y * y; }
    if (MODE == WKV) {
      sw[i] = expf(p.log_decay[(static_cast<long long>(row) * p.H + h) * dk + i]);
      s0 += x * y * ld(p.u + h * dk + i);
    }
  }
  if (MODE == DELTA) {
    s0 = rows::block_sum(s0, red);
    s1 = rows::block_sum(s1, red);
    const float fq = p.scale * rsqrtf(s0 + 1e-6f), fk = rsqrtf(s1 + 1e-6f);
    delta_gates(p, row, h, a, b);               // decay, beta
    for (int i = threadIdx.x; i < dk; i += STEP_THREADS) { sq[i] *= fq; sk[i] *= fk; }
  } else if (MODE == MEMORY) {
    float in, forget;
    memory_gates(p, row, h, in, forget);
    const float m = fresh ? 0.f : p.m[rh], top = fmaxf(forget + m, in);
    a = expf(forget + m - top);
    b = expf(in - top);
    float dot = 0.f;
    for (int i = threadIdx.x; i < dk; i += STEP_THREADS) {
      float* n = p.n + rh * dk + i;
      const float x = (fresh ? 0.f : a * *n) + b * sk[i];
      *n = x;
      sq[i] *= p.scale;
      dot += x * sq[i];
    }
    dot = rows::block_sum(dot, red);            // (every thread has read m by here)
    c = __fdividef(1.f, fmaxf(fabsf(dot), expf(-top)) + 1e-6f);
    if (threadIdx.x == 0) p.m[rh] = top;
  } else {
    c = rows::block_sum(s0, red);               // the bonus
  }
  __syncthreads();
  float* S = p.state + rh * dk * dv;
  for (int t0 = blockIdx.y * TILE; t0 < dv; t0 += gridDim.y * TILE) {
    const int col = t0 + lane * V;
    const bool live = col < dv;                 // V divides dv where V > 1
    float x[U][V], acc[V], vv[V], uu[V];
#pragma unroll
    for (int j = 0; j < V; ++j) { acc[j] = 0.f; vv[j] = live ? ld(v + col + j) : 0.f; uu[j] = vv[j]; }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = group + u * GROUPS;
#pragma unroll
      for (int j = 0; j < V; ++j) x[u][j] = 0.f;
      if (live && i < dk && !fresh) rows::load_v<V>(S + static_cast<long long>(i) * dv + col, x[u]);
    }
    if (MODE == DELTA) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = group + u * GROUPS;
        if (i < dk) {
          const float kk = sk[i];
#pragma unroll
          for (int j = 0; j < V; ++j) acc[j] += kk * x[u][j];
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) part[group * TILE + lane * V + j] = acc[j];
      __syncthreads();
      for (int cc = threadIdx.x; cc < TILE; cc += STEP_THREADS) {
        float s = 0.f;
#pragma unroll
        for (int gg = 0; gg < GROUPS; ++gg) s += part[gg * TILE + cc];
        su[cc] = t0 + cc < dv ? b * (ld(v + t0 + cc) - a * s) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int j = 0; j < V; ++j) { uu[j] = su[lane * V + j]; acc[j] = 0.f; }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = group + u * GROUPS;
      if (live && i < dk) {
        const float kk = MODE == MEMORY ? b * sk[i] : sk[i], qq = sq[i], keep = MODE == WKV ? sw[i] : a;
#pragma unroll
        for (int j = 0; j < V; ++j) {
          if (MODE == WKV) acc[j] += qq * x[u][j];
          x[u][j] = keep * x[u][j] + kk * uu[j];
          if (MODE != WKV) acc[j] += qq * x[u][j];
        }
        rows::store_v<V>(S + static_cast<long long>(i) * dv + col, x[u]);
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) part[group * TILE + lane * V + j] = acc[j];
    __syncthreads();
    for (int cc = threadIdx.x; cc < TILE; cc += STEP_THREADS) {
      float s = 0.f;
#pragma unroll
      for (int gg = 0; gg < GROUPS; ++gg) s += part[gg * TILE + cc];
      if (t0 + cc < dv) st(o + t0 + cc, MODE == MEMORY ? s * c : MODE == WKV ? s + c * ld(v + t0 + cc) : s);
    }
    __syncthreads();
  }
}

// grid (H, ceil(dv / COLS), rows), 4 warps.  RL lanes share a value column, each with KR key rows of it in registers for the whole call; rows are dealt
// in fours.  Tokens go through shared memory TOK at a time, with everything that does not depend on the state made there.
constexpr int SEQ_THREADS = 128;
template <int MODE, typename T, int KR, int RL, int TOK>
__global__ void __launch_bounds__(SEQ_THREADS)
gated_sequence_kernel(Args<T> p) {
  constexpr int DK = KR * RL, CL = 32 / RL, COLS = 4 * CL;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                               // [TOK][DK]
  float* sk = sq + TOK * DK;
  float* sw = sk + TOK * DK;                    // [TOK][DK], wkv
  float* sv = sw + (MODE == WKV ? TOK * DK : 0);   // [TOK][COLS]: values, then outputs
  float* sc = sv + TOK * COLS;                  // [TOK][4]
  const int dk = p.dk, dv = p.dv, S_len = p.S, h = blockIdx.x, row = blockIdx.z, c0 = blockIdx.y * COLS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rl = lane % RL, cl = warp * CL + lane / RL, col = c0 + cl;
  const long long t_row = static_cast<long long>(row) * S_len;
  const int first = p.positions[t_row], len = first < 0 ? 0 : min(p.lengths[row] - first, S_len);
  const int g = h / (p.H / p.G), r = p.row_ids == nullptr ? row : p.row_ids[row];
  const long long rh = static_cast<long long>(r) * p.H + h;
  T* o = p.out + (t_row * p.H + h) * dv;
  const long long o_stride = static_cast<long long>(p.H) * dv;
  float* S = p.state == nullptr ? nullptr : p.state + rh * dk * dv;
  const bool held = S != nullptr && first > 0;
  float x[KR], n[MODE == MEMORY ? KR : 1], m = 0.f;
#pragma unroll
  for (int i = 0; i < KR; ++i) {
    const int kr = ((i / 4) * RL + rl) * 4 + i % 4;
    x[i] = held && kr < dk && col < dv ? S[static_cast<long long>(kr) * dv + col] : 0.f;
    if (MODE == MEMORY) n[i] = held && kr < dk ? p.n_before[rh * dk + kr] : 0.f;
  }
  if (MODE == MEMORY && held) m = p.m_before[rh];
  for (int t0 = 0; t0 < len; t0 += TOK) {
    const int cnt = min(TOK, len - t0);
    __syncthreads();
    for (int i = tid; i < cnt * DK; i += SEQ_THREADS) {
      const int t = i / DK, c = i - t * DK;
      const long long tok = t_row + t0 + t;
      const bool ok = c < dk;
      sq[i] = ok ? ld(p.q + tok * p.q_stride + g * dk + c) * (MODE == MEMORY ? p.scale : 1.f) : 0.f;
      sk[i] = ok ? ld(p.k + tok * p.k_stride + g * dk + c) : 0.f;
      if (MODE == WKV) sw[i] = ok ? expf(p.log_decay[(tok * p.H + h) * dk + c]) : 0.f;
    }
    for (int i = tid; i < cnt * COLS; i += SEQ_THREADS) {
      const int t = i / COLS, c = c0 + i - t * COLS;
      sv[i] = c < dv ? ld(p.v + (t_row + t0 + t) * p.v_stride + h * dv + c) : 0.f;
    }
    __syncthreads();
    if (MODE == MEMORY) {
      if (warp == 0) {                          // lane = token
        static_assert(TOK <= 32, "a lane per token");
        float in = 0.f, forget = 0.f, mine = 0.f, before = 0.f;
        if (lane < cnt) memory_gates(p, t_row + t0 + lane, h, in, forget);
        float run = m;
        for (int t = 0; t < cnt; ++t) {
          const float next = fmaxf(__shfl_sync(0xffffffffu, forget, t) + run, __shfl_sync(0xffffffffu, in, t));
          if (lane == t) { before = run; mine = next; }
          run = next;
        }
        if (lane < cnt) {
          sc[lane * 4] = expf(forget + before - mine);
          sc[lane * 4 + 1] = expf(in - mine);
          sc[lane * 4 + 2] = expf(-mine);
          sc[lane * 4 + 3] = mine;
        }
      }
    } else {
      for (int t = warp; t < cnt; t += 4) {     // a warp per token
        float s0 = 0.f, s1 = 0.f;
        for (int c = lane; c < dk; c += 32) {
          const float a = sq[t * DK + c], b = sk[t * DK + c];
          if (MODE == DELTA) { s0 += a * a; s1 += b * b; }
          else s0 += a * b * ld(p.u + h * dk + c);
        }
#pragma unroll
        for (int q = 16; q > 0; q >>= 1) { s0 += __shfl_xor_sync(0xffffffffu, s0, q); s1 += __shfl_xor_sync(0xffffffffu, s1, q); }
        if (MODE == DELTA) {
          const float fq = p.scale * rsqrtf(s0 + 1e-6f), fk = rsqrtf(s1 + 1e-6f);
          for (int c = lane; c < dk; c += 32) { sq[t * DK + c] *= fq; sk[t * DK + c] *= fk; }
          if (lane == 0) delta_gates(p, t_row + t0 + t, h, sc[t * 4], sc[t * 4 + 1]);
        } else if (lane == 0) {
          sc[t * 4] = s0;
        }
      }
    }
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {
      const float a = sc[t * 4], b = sc[t * 4 + 1], v = sv[t * COLS + cl];
      float4 kk[KR / 4];
#pragma unroll
      for (int i = 0; i < KR / 4; ++i) kk[i] = *reinterpret_cast<const float4*>(sk + t * DK + (i * RL + rl) * 4);
      float add = v;
      if (MODE == DELTA) {
        float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < KR / 4; ++i) {
          s[0] += kk[i].x * x[4 * i]; s[1] += kk[i].y * x[4 * i + 1];
          s[2] += kk[i].z * x[4 * i + 2]; s[3] += kk[i].w * x[4 * i + 3];
        }
        float dot = (s[0] + s[1]) + (s[2] + s[3]);
#pragma unroll
        for (int q = RL / 2; q > 0; q >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, q);
        add = b * (v - a * dot);
      }
      float acc[4] = {0.f, 0.f, 0.f, 0.f}, den = 0.f;
#pragma unroll
      for (int i = 0; i < KR / 4; ++i) {
        const float4 qq = *reinterpret_cast<const float4*>(sq + t * DK + (i * RL + rl) * 4);
        const float4 ww = MODE == WKV ? *reinterpret_cast<const float4*>(sw + t * DK + (i * RL + rl) * 4) : make_float4(a, a, a, a);
        const float ke[4] = {kk[i].x, kk[i].y, kk[i].z, kk[i].w}, qe[4] = {qq.x, qq.y, qq.z, qq.w}, we[4] = {ww.x, ww.y, ww.z, ww.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int at = 4 * i + e;
          if (MODE == WKV) acc[e] += qe[e] * x[at];
          const float w = MODE == MEMORY ? b * ke[e] : ke[e];
          x[at] = we[e] * x[at] + w * add;
          if (MODE != WKV) acc[e] += qe[e] * x[at];
          if (MODE == MEMORY) { n[at] = a * n[at] + w; den += qe[e] * n[at]; }
        }
      }
      float out = (acc[0] + acc[1]) + (acc[2] + acc[3]);
#pragma unroll
      for (int q = RL / 2; q > 0; q >>= 1) {
        out += __shfl_xor_sync(0xffffffffu, out, q);
        if (MODE == MEMORY) den += __shfl_xor_sync(0xffffffffu, den, q);
      }
      if (MODE == WKV) out += a * v;
      if (MODE == MEMORY) out = __fdividef(out, fmaxf(fabsf(den), sc[t * 4 + 2]) + 1e-6f);
      if (rl == 0) sv[t * COLS + cl] = out;     // (the column's lanes have read their value: the shuffles stand between)
    }
    if (MODE == MEMORY) m = sc[(cnt - 1) * 4 + 3];
    __syncthreads();
    for (int i = tid; i < cnt * COLS; i += SEQ_THREADS) {
      const int t = i / COLS, c = c0 + i - t * COLS;
      if (c < dv) st(o + (t0 + t) * o_stride + c, sv[i]);
    }
  }
  for (int i = tid; i < (S_len - len) * COLS; i += SEQ_THREADS) {
    const int t = len + i / COLS, c = c0 + i % COLS;
    if (c < dv) st(o + t * o_stride + c, 0.f);
  }
  if (S == nullptr || len == 0) return;
#pragma unroll
  for (int i = 0; i < KR; ++i) {
    const int kr = ((i / 4) * RL + rl) * 4 + i % 4;
    if (kr < dk && col < dv) S[static_cast<long long>(kr) * dv + col] = x[i];
    if (MODE == MEMORY && blockIdx.y == 0 && warp == 0 && lane < RL && kr < dk) p.n[rh * dk + kr] = n[i];
  }
  if (MODE == MEMORY && blockIdx.y == 0 && tid == 0) p.m[rh] = m;
}

template <int MODE, typename T, int V, int LANES, int U>
int step_go(const Args<T>& p, cudaStream_t stream) {
  constexpr int GROUPS = STEP_THREADS / LANES, TILE = LANES * V;
  const size_t smem = static_cast<size_t>((MODE == WKV ? 3 : 2) * p.dk + GROUPS * TILE + TILE) * 4;
  const int tiles = (p.dv + TILE - 1) / TILE;
  gated_step_kernel<MODE, T, V, LANES, U><<<dim3(p.H, MODE == MEMORY ? 1 : tiles, p.R), STEP_THREADS, smem, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <int MODE, typename T>
int step_any(const Args<T>& p, cudaStream_t stream) {
  const int dk = p.dk;
  if (p.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(p.state) & 15) == 0) {
    // wide tiles once there are blocks enough for every SM
    if (p.dv > 32 && dk <= 128 && static_cast<long long>(p.R) * p.H >= 592) return dk <= 64 ? step_go<MODE, T, 4, 32, 8>(p, stream) : step_go<MODE, T, 4, 32, 16>(p, stream);
    if (dk <= 64) return step_go<MODE, T, 4, 8, 2>(p, stream);
    if (dk <= 128) return step_go<MODE, T, 4, 8, 4>(p, stream);
    if (dk <= 256) return step_go<MODE, T, 4, 8, 8>(p, stream);
    if (dk <= 512) return step_go<MODE, T, 4, 8, 16>(p, stream);
    return -3;
  }
  if (dk <= 32) return step_go<MODE, T, 1, 32, 4>(p, stream);
  if (dk <= 128) return step_go<MODE, T, 1, 32, 16>(p, stream);
  if (dk <= 512) return step_go<MODE, T, 1, 32, 64>(p, stream);
  return -3;
}

template <int MODE, typename T, int KR, int RL, int TOK>
int seq_go(const Args<T>& p, cudaStream_t stream) {
  constexpr int COLS = 4 * (32 / RL);
  const size_t smem = static_cast<size_t>(TOK) * ((MODE == WKV ? 3 : 2) * KR * RL + COLS + 4) * 4;
  cudaError_t e = cudaFuncSetAttribute(gated_sequence_kernel<MODE, T, KR, RL, TOK>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  gated_sequence_kernel<MODE, T, KR, RL, TOK><<<dim3(p.H, (p.dv + COLS - 1) / COLS, p.R), SEQ_THREADS, smem, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <int MODE, typename T>
int seq_any(const Args<T>& p, cudaStream_t stream) {
  const int dk = p.dk;
  if (dk <= 16) return seq_go<MODE, T, 16, 1, 32>(p, stream);
  if (dk <= 32) return seq_go<MODE, T, 16, 2, 32>(p, stream);
  if (dk <= 64) return seq_go<MODE, T, 16, 4, 32>(p, stream);
  if (dk <= 128) return seq_go<MODE, T, 32, 4, 32>(p, stream);
  if (dk <= 256) return seq_go<MODE, T, 32, 8, 16>(p, stream);
  if (dk <= 512) return seq_go<MODE, T, 32, 16, 16>(p, stream);
  return -3;
}

template <int MODE, typename T>
int run(const Args<T>& p, cudaStream_t stream) {
  return p.S == 1 && p.state != nullptr ? step_any<MODE, T>(p, stream) : seq_any<MODE, T>(p, stream);
}

template <typename T>
int any(int mode, const Args<T>& p, cudaStream_t stream) {
  if (mode == DELTA) return run<DELTA, T>(p, stream);
  if (mode == MEMORY) return run<MEMORY, T>(p, stream);
  return run<WKV, T>(p, stream);
}

}  // namespace gated
}  // namespace dewb

using namespace dewb::gated;

// One token per row (S 1, with a state) or a call's tokens one after another.
extern "C" int dewb_gated_recurrence(int mode, const dewb_gated_args* a, int fp32, void* stream_ptr) {
  if (a == nullptr) return -3;
  if (a->R <= 0 || a->S <= 0) return 0;
  if (!args_ok(mode, *a)) return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  return fp32 ? any<float>(mode, Args<float>(*a), stream) : any<bf16>(mode, Args<bf16>(*a), stream);
}
