// What the kernels of the token-gated recurrences share: their arguments and the gates of a token.
#pragma once
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "rows.cuh"

// q, k [tokens, G dk] and v [tokens, H dv] in rows of their own strides (elements).  Null where a mode or a call has none: state (nothing kept), n / m and
// n_before / m_before (what the call started from, where several blocks read it while one writes), gates, log_decay, u, row_ids.
extern "C" struct dewb_gated_args {
  const void *q, *k, *v;
  long long q_stride, k_stride, v_stride;
  const float* gates;          // [tokens, 2 H]: delta b | a, memory zi | zf
  const float *bias0, *bias1;  // [H]: delta A_log, dt_bias; memory bi, bf
  const float* log_decay;      // [tokens, H dk]: wkv
  const void* u;               // [H, dk]: wkv
  float *state, *n, *m;        // [store rows, H, dk, dv], [store rows, H, dk], [store rows, H]
  const float *n_before, *m_before;
  const int *positions, *lengths, *row_ids;
  void* out;                   // [tokens, H, dv]
  float scale, cap;
  int R, S, H, G, dk, dv;
};

namespace dewb {
namespace gated {

using rows::bf16;
enum : int { DELTA = 0, MEMORY = 1, WKV = 2 };

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }

template <typename T>
struct Args {
  const T *q, *k, *v;
  long long q_stride, k_stride, v_stride;
  const float *gates, *bias0, *bias1, *log_decay;
  const T* u;
  float *state, *n, *m;
  const float *n_before, *m_before;
  const int *positions, *lengths, *row_ids;
  T* out;
  float scale, cap;
  int R, S, H, G, dk, dv;
  explicit Args(const dewb_gated_args& a)
      : q(static_cast<const T*>(a.q)), k(static_cast<const T*>(a.k)), v(static_cast<const T*>(a.v)), q_stride(a.q_stride), k_stride(a.k_stride),
        v_stride(a.v_stride), gates(a.gates), bias0(a.bias0), bias1(a.bias1), log_decay(a.log_decay), u(static_cast<const T*>(a.u)), state(a.state), n(a.n),
        m(a.m), n_before(a.n_before), m_before(a.m_before), positions(a.positions), lengths(a.lengths), row_ids(a.row_ids), out(static_cast<T*>(a.out)),
        scale(a.scale), cap(a.cap), R(a.R), S(a.S), H(a.H), G(a.G), dk(a.dk), dv(a.dv) {}
};

inline bool args_ok(int mode, const dewb_gated_args& a) {
  if (mode < DELTA || mode > WKV || a.H < 1 || a.G < 1 || a.H % a.G || a.dk < 1 || a.dv < 1 || a.R > 65535) return false;
  if (a.q_stride < static_cast<long long>(a.G) * a.dk || a.k_stride < static_cast<long long>(a.G) * a.dk || a.v_stride < static_cast<long long>(a.H) * a.dv) return false;
  if (a.positions == nullptr || a.lengths == nullptr || a.out == nullptr) return false;
  if (mode == WKV) return a.log_decay != nullptr && a.u != nullptr && a.G == a.H;
  if (a.gates == nullptr || a.bias0 == nullptr || a.bias1 == nullptr) return false;
  if (mode == DELTA) return true;
  return a.G == a.H && a.cap > 0.f && (a.state == nullptr || (a.n != nullptr && a.m != nullptr && (a.S == 1 || (a.n_before != nullptr && a.m_before != nullptr))));
}

// ln(1 + e^x)
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// The logarithm of a head's decay, and its step.
template <typename T>
__device__ __forceinline__ void delta_log_gates(const Args<T>& p, int h, float zb, float za, float& log_decay, float& beta) {
  beta = __fdividef(1.f, 1.f + expf(-zb));
  log_decay = -expf(p.bias0[h]) * softplus(za + p.bias1[h]);
}
template <typename T>
__device__ __forceinline__ void delta_gates(const Args<T>& p, long long token, int h, float& decay, float& beta) {
  const float* z = p.gates + token * 2 * p.H + h;
  delta_log_gates(p, h, z[0], z[p.H], decay, beta);
  decay = expf(decay);
}

// Logarithms of the input and the forget gate.
template <typename T>
__device__ __forceinline__ void memory_gates(const Args<T>& p, int h, float zi, float zf, float& in, float& forget) {
  const float inv = __fdividef(1.f, p.cap);
  in = p.cap * tanhf((zi + p.bias0[h]) * inv);
  forget = -softplus(-p.cap * tanhf((zf + p.bias1[h]) * inv));
}
template <typename T>
__device__ __forceinline__ void memory_gates(const Args<T>& p, long long token, int h, float& in, float& forget) {
  const float* z = p.gates + token * 2 * p.H + h;
  memory_gates(p, h, z[0], z[p.H], in, forget);
}

}  // namespace gated
}  // namespace dewb
