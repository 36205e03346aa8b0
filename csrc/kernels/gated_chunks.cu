// The recurrences of gated_recurrence.cu over a call's tokens in chunks on the tensor cores, for sm_100a (bf16, dk up to 128, widths in multiples of 8).
//
// One block walks a (row, head, 64 or 128 value columns) chunk by chunk, the next chunk's rows on their way (cp.async).  A warp keeps the state of 16 value columns, transposed ([value, key], fp32
// accumulators) for the whole call: a fragment of it turns into an operand without leaving the registers, and once a chunk's scores lie in shared memory a warp
// needs nothing from the others.  Everything that is not a bf16 activation - the state, decayed scores, what the delta rule writes - enters its products as a
// pair of bf16 (value and rounding rest: 16 bits of mantissa); weights of a token or a channel are fp32 factors.  No exponent is above 0 by construction.
//
//   gated_chunks   64 tokens.  memory: with F the sums of the log forget gates and g_j = i_j - F_j, the running maximum is F_i + M_i, M_i = max(m, g_0 .. g_i);
//                      o_i = [e^(m - M_i) S^T q_i + sum_{j <= i} e^(g_j - M_i) (q_i . k_j) v_j] / (the same sums with 1 for v, bounded below, + 1e-6)
//                  delta: with G the sums of the log decays and A_ij = beta_i e^(G_i - G_j) (k_i . k_j) below the diagonal, the chunk's writes U solve
//                      (I + A) U = beta (V - e^G K S),   o = e^G Q S + [(q_i . k_j) e^(G_i - G_j)]_{j <= i} U,   S' = e^G_n S + (e^(G_n - G) K)^T U
//                  by blocks of 16: the diagonal blocks are inverted, the rest is substitution
//   wkv_chunks     16 tokens, as the decays differ from channel to channel: products of a token pair are formed channel by channel with their own exponent
//
// Compiled without fast math.
#include <cstdint>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../common/gated_rule.cuh"
#include "../common/mma_bf16.cuh"

namespace dewb {
namespace gated {

using namespace mma16;

constexpr int CT = 64;              // tokens per chunk

template <int MODE, int DK, int NW>
struct ChunkSmem {
  static constexpr int VT = NW * 16;
  bf16 q[2][CT][DK + 8], k[2][CT][DK + 8], v[2][CT][VT + 8];  // two stages
  bf16 p[2][CT][CT + 8];                                     // scores as the outputs take them: value, rest
  bf16 a[MODE == DELTA ? 2 : 1][MODE == DELTA ? CT : 1][CT + 8];   // delta: -A below the diagonal blocks
  bf16 t[2][4][16][MODE == DELTA ? 24 : 8];                  // delta: the diagonal blocks of (I + A)^-1
  float diag[MODE == DELTA ? 4 : 1][16][16];                 // ... of A, by columns
  float x0[CT], x1[CT], x2[CT], x3[CT], x4[CT], x5[CT], x6[CT];   // of the tokens, see below
  float part[MODE == MEMORY ? CT : 1][4];                    // memory: sums of a row's scores, by block of 16 keys
  float n[MODE == MEMORY ? NW * 32 : 1];                     // memory: the normaliser, in the parts their threads own
  float end[2];
};

// 16 bytes of a token's row, zeros past its columns
__device__ __forceinline__ uint4 row16(const bf16* p, bool ok) { return ok ? *reinterpret_cast<const uint4*>(p) : make_uint4(0, 0, 0, 0); }

// 16 bytes into shared memory, zeros where there is nothing to read (the address has to be valid all the same)
__device__ __forceinline__ void cp16(void* dst, const void* src, bool live) {
  const int n = live ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(n) : "memory");
}

// d += a b for two tiles of eight columns, b [16, 16]
__device__ __forceinline__ void mma2(float (&d0)[4], float (&d1)[4], const uint32_t (&a)[4], const uint32_t (&b)[4]) {
  mma(d0, a, b[0], b[1]);
  mma(d1, a, b[2], b[3]);
}

// c [16 values, 16 tokens] as an operand whose rows are values and whose reduction runs over the tokens
__device__ __forceinline__ void as_operand(const float (&lo)[4], const float (&hi)[4], uint32_t (&big)[4], uint32_t (&rest)[4]) {
  split2(lo[0], lo[1], big[0], rest[0]);
  split2(lo[2], lo[3], big[1], rest[1]);
  split2(hi[0], hi[1], big[2], rest[2]);
  split2(hi[2], hi[3], big[3], rest[3]);
}

__device__ __forceinline__ float warp_scan(float v, int lane) {
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float u = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v += u;
  }
  return v;
}
__device__ __forceinline__ float warp_max_scan(float v, int lane) {
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float u = __shfl_up_sync(0xffffffffu, v, o);
    if (lane >= o) v = fmaxf(v, u);
  }
  return v;
}

// grid (H, ceil(dv / VT), rows), NW warps
template <int MODE, int DK, int NW>
__global__ void __launch_bounds__(NW * 32, NW == 4 ? 2 : 1)
gated_chunks_kernel(Args<bf16> p) {
  extern __shared__ __align__(16) uint8_t raw[];
  ChunkSmem<MODE, DK, NW>& sm = *reinterpret_cast<ChunkSmem<MODE, DK, NW>*>(raw);
  constexpr int CTHREADS = NW * 32, VT = NW * 16;
  constexpr int NK = DK / 8;                       // 8-column tiles of the state
  const int dk = p.dk, dv = p.dv, S_len = p.S, h = blockIdx.x, row = blockIdx.z, c0 = blockIdx.y * VT;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, lg = lane >> 2, t2 = (lane & 3) * 2;
  const long long t_row = static_cast<long long>(row) * S_len;
  const int first = p.positions[t_row], len = first < 0 ? 0 : min(p.lengths[row] - first, S_len);
  const int gk = h / (p.H / p.G), r = p.row_ids == nullptr ? row : p.row_ids[row];
  const long long rh = static_cast<long long>(r) * p.H + h;
  const bf16 *qb = p.q + t_row * p.q_stride + gk * dk, *kb = p.k + t_row * p.k_stride + gk * dk, *vb = p.v + t_row * p.v_stride + h * dv + c0;
  bf16* o = p.out + (t_row * p.H + h) * dv + c0;
  const long long o_stride = static_cast<long long>(p.H) * dv;
  float* S = p.state == nullptr ? nullptr : p.state + rh * dk * dv;
  const bool held = S != nullptr && first > 0;
  const int w0 = warp * 16;                        // this warp's value columns
  float st_acc[NK][4];
#pragma unroll
  for (int n = 0; n < NK; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int kr = n * 8 + t2 + (e & 1), vc = c0 + w0 + lg + (e >> 1) * 8;
      st_acc[n][e] = held && kr < dk && vc < dv ? S[static_cast<long long>(kr) * dv + vc] : 0.f;
    }
  float m = MODE == MEMORY && held ? p.m_before[rh] : 0.f;
  if (MODE == MEMORY)
    for (int i = tid; i < CTHREADS; i += CTHREADS) sm.n[i] = held && i < dk ? p.n_before[rh * dk + i] : 0.f;
  const int vcols = min(VT, dv - c0);
  auto fetch = [&](int t0, int s) {
    constexpr int PK = DK / 8, PV = VT / 8;        // 16-byte pieces of a row
    const int ck = (tid % PK) * 8, cv = (tid % PV) * 8;
#pragma unroll
    for (int t = tid / PK; t < CT; t += CTHREADS / PK) {
      const bool ok = t0 + t < len && ck < dk;
      cp16(&sm.q[s][t][ck], ok ? qb + (t0 + t) * p.q_stride + ck : p.q, ok);
      cp16(&sm.k[s][t][ck], ok ? kb + (t0 + t) * p.k_stride + ck : p.k, ok);
    }
#pragma unroll
    for (int t = tid / PV; t < CT; t += CTHREADS / PV) {
      const bool ok = t0 + t < len && cv < vcols;
      cp16(&sm.v[s][t][cv], ok ? vb + (t0 + t) * p.v_stride + cv : p.v, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // the first warp's gates, a chunk ahead: tokens lane and lane + 32
  float z0[2] = {0.f, 0.f}, z1[2] = {0.f, 0.f};
  auto gates = [&](int t0) {
#pragma unroll
    for (int x = 0; x < 2; ++x)
      if (t0 + lane + 32 * x < len) {
        const float* z = p.gates + (t_row + t0 + lane + 32 * x) * 2 * p.H + h;
        z0[x] = z[0];
        z1[x] = z[p.H];
      }
  };
  if (len > 0) {
    fetch(0, 0);
    if (warp == 0) gates(0);
  }
  for (int t0 = 0, stage = 0; t0 < len; t0 += CT, stage ^= 1) {
    const int n = min(CT, len - t0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                               // this chunk is there, the one before has been read
    if (t0 + CT < len) fetch(t0 + CT, stage ^ 1);
    const bf16 (&sq_)[CT][DK + 8] = sm.q[stage], (&sk_)[CT][DK + 8] = sm.k[stage];
    bf16 (&sv_)[CT][VT + 8] = sm.v[stage];
    // ---- scalars of the tokens.  memory: x0 = g, x1 = M, x2 = scale e^(m - M), x3 = e^-(F + M), x4 = q . n, x5 = e^(g - M_end);
    //      delta: x0 = beta, x1 = G, x2, x3 = factors of q and k, x4 = x2 e^G, x5 = x3 e^(G_end - G), x6 = beta x3 e^G
    {
      constexpr int PER = CTHREADS / CT, PARTS = CTHREADS / DK;        // threads per token; parts of the normaliser
      const int t = tid / PER, c0_ = (tid % PER) * 8;
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int c = c0_; c < DK; c += 8 * PER) {
        float a[8], b[8];
        rows::load_v<8>(&sq_[t][c], a);
        if (MODE == DELTA) rows::load_v<8>(&sk_[t][c], b);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          if (MODE == DELTA) {
            s0 += a[j] * a[j];
            s1 += b[j] * b[j];
          } else {
#pragma unroll
            for (int x = 0; x < PARTS; ++x) s0 += a[j] * sm.n[x * DK + c + j];
          }
        }
      }
#pragma unroll
      for (int x = PER / 2; x > 0; x >>= 1) {
        s0 += __shfl_xor_sync(0xffffffffu, s0, x);
        s1 += __shfl_xor_sync(0xffffffffu, s1, x);
      }
      if (tid % PER == 0) {
        if (MODE == DELTA) { sm.x2[t] = p.scale * rsqrtf(s0 + 1e-6f); sm.x3[t] = rsqrtf(s1 + 1e-6f); }
        else sm.x4[t] = s0;
      }
    }
    if (warp == 0) {
      float a[2], b[2];                            // beta or log input gate; log decay or log forget gate
#pragma unroll
      for (int x = 0; x < 2; ++x) {                // what lies past the end neither writes nor forgets
        a[x] = MODE == MEMORY ? -INFINITY : 0.f;
        b[x] = 0.f;
        if (lane + 32 * x < n) {
          if (MODE == MEMORY) memory_gates(p, h, z0[x], z1[x], a[x], b[x]);
          else delta_log_gates(p, h, z0[x], z1[x], b[x], a[x]);
        }
      }
      gates(t0 + CT);
      const float F0 = warp_scan(b[0], lane), F1 = warp_scan(b[1], lane) + __shfl_sync(0xffffffffu, F0, 31);
      if (MODE == DELTA) {
        sm.x0[lane] = a[0]; sm.x0[lane + 32] = a[1];
        sm.x1[lane] = F0; sm.x1[lane + 32] = F1;
      } else {
        const float g0 = a[0] - F0, g1 = a[1] - F1;
        const float M0 = fmaxf(m, warp_max_scan(g0, lane)), M1 = fmaxf(__shfl_sync(0xffffffffu, M0, 31), warp_max_scan(g1, lane));
        sm.x0[lane] = g0; sm.x0[lane + 32] = g1;
        sm.x1[lane] = M0; sm.x1[lane + 32] = M1;
        sm.x2[lane] = p.scale * expf(m - M0); sm.x2[lane + 32] = p.scale * expf(m - M1);
        sm.x3[lane] = expf(-(F0 + M0)); sm.x3[lane + 32] = expf(-(F1 + M1));
        if (lane == 31) { sm.end[0] = M1; sm.end[1] = F1 + M1; }
      }
    }
    __syncthreads();
    if (tid < CT) {
      if (MODE == MEMORY) {
        sm.x5[tid] = expf(sm.x0[tid] - sm.end[0]);
      } else {
        const float e = expf(sm.x1[tid]), fk = sm.x3[tid];
        sm.x4[tid] = sm.x2[tid] * e;
        sm.x5[tid] = fk * expf(sm.x1[CT - 1] - sm.x1[tid]);
        sm.x6[tid] = sm.x0[tid] * fk * e;
      }
    }
    // ---- scores: the ten 16 x 16 blocks on and below the diagonal, the diagonal ones first
    // (eight warps: a diagonal one each for four of them, the others deal out the rest)
    for (int blk = warp; blk < 10; blk += NW == 8 && warp < 4 ? 10 : 4) {
      const int off = blk - 4;                     // 0..5: (1,0) (2,0) (2,1) (3,0) (3,1) (3,2)
      const int bi = blk < 4 ? blk : off < 1 ? 1 : off < 3 ? 2 : 3, bj = blk < 4 ? blk : off < 1 ? 0 : off < 3 ? off - 1 : off - 3;
      const int i0 = bi * 16, j0 = bj * 16;
      float sq[2][4], sk[2][4];
      {
        float s[2][2][4] = {}, z[2][2][4] = {};    // even and odd steps apart: their products do not wait for each other
#pragma unroll
        for (int kk = 0; kk < DK; kk += 16) {
          uint32_t qa[4], ka[4], b[4];
          ldsm4(b, smem_addr(&sk_[j0 + (lane & 7) + (lane >> 4) * 8][kk + ((lane >> 3) & 1) * 8]));
          ldsm4(qa, smem_addr(&sq_[i0 + (lane & 15)][kk + (lane >> 4) * 8]));
          mma2(s[kk / 16 & 1][0], s[kk / 16 & 1][1], qa, b);
          if (MODE == DELTA) {
            ldsm4(ka, smem_addr(&sk_[i0 + (lane & 15)][kk + (lane >> 4) * 8]));
            mma2(z[kk / 16 & 1][0], z[kk / 16 & 1][1], ka, b);
          }
        }
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
          for (int e = 0; e < 4; ++e) { sq[x][e] = s[0][x][e] + s[1][x][e]; sk[x][e] = z[0][x][e] + z[1][x][e]; }
      }
      float sum[2] = {0.f, 0.f};
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = i0 + lg + 8 * e, j = j0 + half * 8 + t2;
          float x[2], y[2];
#pragma unroll
          for (int z = 0; z < 2; ++z) {
            const bool on = j + z <= i;
            if (MODE == MEMORY) {
              x[z] = on ? sq[half][2 * e + z] * p.scale * __expf(sm.x0[j + z] - sm.x1[i]) : 0.f;
              sum[e] += x[z];
            } else {
              const float w = on ? sm.x3[j + z] * __expf(sm.x1[i] - sm.x1[j + z]) : 0.f;
              x[z] = sq[half][2 * e + z] * w * sm.x2[i];
              y[z] = j + z < i ? sk[half][2 * e + z] * w * sm.x3[i] * sm.x0[i] : 0.f;
            }
          }
          uint32_t big, rest;
          split2(x[0], x[1], big, rest);
          *reinterpret_cast<uint32_t*>(&sm.p[0][i][j]) = big;
          *reinterpret_cast<uint32_t*>(&sm.p[1][i][j]) = rest;
          if constexpr (MODE == DELTA) {
            if (bi == bj) {
              sm.diag[bi][j - j0][i - i0] = y[0];
              sm.diag[bi][j - j0 + 1][i - i0] = y[1];
            } else {
              split2(-y[0], -y[1], big, rest);
              *reinterpret_cast<uint32_t*>(&sm.a[0][i][j]) = big;
              *reinterpret_cast<uint32_t*>(&sm.a[1][i][j]) = rest;
            }
          }
        }
      if constexpr (MODE == MEMORY) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
          sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
          if ((lane & 3) == 0) sm.part[i0 + lg + 8 * e][bj] = sum[e];
        }
      } else if (bi == bj) {                       // the block's inverse, a column per lane
        __syncwarp();
        float x[16];
        const int c = lane & 15;
#pragma unroll
        for (int i = 0; i < 16; ++i) x[i] = i == c ? 1.f : 0.f;
#pragma unroll
        for (int j = 0; j < 15; ++j)
#pragma unroll
          for (int i = (j + 1) & ~3; i < 16; i += 4) {
            const float4 d = *reinterpret_cast<const float4*>(&sm.diag[bi][j][i]);      // (zeros on and above the diagonal)
            x[i] -= d.x * x[j]; x[i + 1] -= d.y * x[j]; x[i + 2] -= d.z * x[j]; x[i + 3] -= d.w * x[j];
          }
        if (lane < 16) {
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const bf16 b = __float2bfloat16(x[i]);
            sm.t[0][bi][i][c] = b;
            sm.t[1][bi][i][c] = __float2bfloat16(x[i] - __bfloat162float(b));
          }
        }
      }
    }
    __syncthreads();
    // ---- from the state, transposed: S^T Q^T (and S^T K^T), [16 values, 64 tokens]
    float acc[8][4], u[MODE == DELTA ? 8 : 1][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
      if (MODE == DELTA) u[MODE == DELTA ? j : 0][0] = u[MODE == DELTA ? j : 0][1] = u[MODE == DELTA ? j : 0][2] = u[MODE == DELTA ? j : 0][3] = 0.f;
    }
#pragma unroll
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t big[4], rest[4];
      as_operand(st_acc[kk / 8], st_acc[kk / 8 + 1], big, rest);
      auto rows_at = [&](const bf16 (&m)[CT][DK + 8], int j, uint32_t (&b)[4]) {
        ldsm4(b, smem_addr(&m[j * 16 + (lane & 7) + (lane >> 4) * 8][kk + ((lane >> 3) & 1) * 8]));
      };
      if constexpr (MODE == DELTA) {               // eight sums between a product and the next one into the same sum
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          uint32_t b0[4], b1[4], c0_[4], c1[4];
          rows_at(sq_, j, b0);
          rows_at(sk_, j, c0_);
          rows_at(sq_, j + 1, b1);
          rows_at(sk_, j + 1, c1);
          mma2(acc[2 * j], acc[2 * j + 1], big, b0);
          mma2(u[2 * j], u[2 * j + 1], big, c0_);
          mma2(acc[2 * j + 2], acc[2 * j + 3], big, b1);
          mma2(u[2 * j + 2], u[2 * j + 3], big, c1);
          mma2(acc[2 * j], acc[2 * j + 1], rest, b0);
          mma2(u[2 * j], u[2 * j + 1], rest, c0_);
          mma2(acc[2 * j + 2], acc[2 * j + 3], rest, b1);
          mma2(u[2 * j + 2], u[2 * j + 3], rest, c1);
        }
      } else {
        uint32_t b[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) rows_at(sq_, j, b[j]);
#pragma unroll
        for (int j = 0; j < 4; ++j) mma2(acc[2 * j], acc[2 * j + 1], big, b[j]);
#pragma unroll
        for (int j = 0; j < 4; ++j) mma2(acc[2 * j], acc[2 * j + 1], rest, b[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int z = 0; z < 2; ++z) {
        const int i = j * 8 + t2 + z;
        const float w = MODE == MEMORY ? sm.x2[i] : sm.x4[i];
        acc[j][z] *= w;
        acc[j][z + 2] *= w;
      }
    if constexpr (MODE == DELTA) {
      // ---- the writes: right-hand sides, then block after block
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        uint32_t vt[4];
        ldsm4_t(vt, smem_addr(&sv_[b * 16 + (lane & 7) + (lane >> 4) * 8][w0 + ((lane >> 3) & 1) * 8]));
#pragma unroll
        for (int x = 0; x < 4; ++x) {              // (an operand of values over tokens has the places of a result)
          float (&d)[4] = u[2 * b + (x >> 1)];
          const int i = b * 16 + (x >> 1) * 8 + t2, e = (x & 1) * 2;
#pragma unroll
          for (int z = 0; z < 2; ++z)
            d[e + z] = sm.x0[i + z] * (z ? hi_f(vt[x]) : lo_f(vt[x])) - sm.x6[i + z] * d[e + z];
        }
      }
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        uint32_t big[4], rest[4];
        auto block = [&](const bf16 (&m)[CT][CT + 8], int i, uint32_t (&x)[4]) {
          ldsm4(x, smem_addr(&m[i * 16 + (lane & 7) + (lane >> 4) * 8][b * 16 + ((lane >> 3) & 1) * 8]));
        };
        {
          uint32_t x[4], y[4];
          float d[2][4] = {}, e[2][4] = {}, f[2][4] = {};
          ldsm4(x, smem_addr(&sm.t[0][b][(lane & 7) + (lane >> 4) * 8][((lane >> 3) & 1) * 8]));
          ldsm4(y, smem_addr(&sm.t[1][b][(lane & 7) + (lane >> 4) * 8][((lane >> 3) & 1) * 8]));
          as_operand(u[2 * b], u[2 * b + 1], big, rest);
          mma2(d[0], d[1], big, x);
          mma2(e[0], e[1], rest, x);
          mma2(f[0], f[1], big, y);
#pragma unroll
          for (int z = 0; z < 2; ++z)
#pragma unroll
            for (int q = 0; q < 4; ++q) u[2 * b + z][q] = d[z][q] + (e[z][q] + f[z][q]);
        }
        as_operand(u[2 * b], u[2 * b + 1], big, rest);
        // what the block means for the later right-hand sides, then for the outputs
#pragma unroll
        for (int i = b + 1; i < 4; ++i) {
          uint32_t x[4], y[4];
          block(sm.a[0], i, x);
          block(sm.a[1], i, y);
          mma2(u[2 * i], u[2 * i + 1], big, x);
          mma2(u[2 * i], u[2 * i + 1], rest, x);
          mma2(u[2 * i], u[2 * i + 1], big, y);
        }
#pragma unroll
        for (int i = b; i < 4; ++i) {
          uint32_t x[4], y[4];
          block(sm.p[0], i, x);
          block(sm.p[1], i, y);
          mma2(acc[2 * i], acc[2 * i + 1], big, x);
          mma2(acc[2 * i], acc[2 * i + 1], rest, x);
          mma2(acc[2 * i], acc[2 * i + 1], big, y);
        }
      }
    }
    if constexpr (MODE == MEMORY) {                // ---- from the chunk: values times scores
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        uint32_t vt[4], x[4][4];
        ldsm4_t(vt, smem_addr(&sv_[b * 16 + (lane & 7) + (lane >> 4) * 8][w0 + ((lane >> 3) & 1) * 8]));
#pragma unroll
        for (int part = 0; part < 2; ++part) {
#pragma unroll
          for (int i = b; i < 4; ++i) ldsm4(x[i], smem_addr(&sm.p[part][i * 16 + (lane & 7) + (lane >> 4) * 8][b * 16 + ((lane >> 3) & 1) * 8]));
#pragma unroll
          for (int i = b; i < 4; ++i) mma2(acc[2 * i], acc[2 * i + 1], vt, x[i]);
        }
      }
    }
    // ---- the state after the chunk
    const float last = MODE == MEMORY ? sm.end[0] : sm.x1[CT - 1];
    const float keep = MODE == MEMORY ? expf(m - last) : expf(last);
#pragma unroll
    for (int j = 0; j < NK; ++j) { st_acc[j][0] *= keep; st_acc[j][1] *= keep; st_acc[j][2] *= keep; st_acc[j][3] *= keep; }
#pragma unroll
    for (int b = 0; b < 4; ++b) {
      if (b * 16 < n) {
        uint32_t big[4], rest[4];
        const int i = b * 16 + t2;
        if constexpr (MODE == MEMORY) {
          uint32_t vt[4];
          ldsm4_t(vt, smem_addr(&sv_[b * 16 + (lane & 7) + (lane >> 4) * 8][w0 + ((lane >> 3) & 1) * 8]));
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int j = i + (x >> 1) * 8;
            split2(lo_f(vt[x]) * sm.x5[j], hi_f(vt[x]) * sm.x5[j + 1], big[x], rest[x]);
          }
        } else {
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int j = i + (x >> 1) * 8, e = (x & 1) * 2;
            const float (&d)[4] = u[2 * b + (x >> 1)];
            split2(d[e] * sm.x5[j], d[e + 1] * sm.x5[j + 1], big[x], rest[x]);
          }
        }
#pragma unroll
        for (int j = 0; j < NK / 2; j += 4) {
          uint32_t x[4][4];
#pragma unroll
          for (int z = 0; z < 4; ++z) ldsm4_t(x[z], smem_addr(&sk_[b * 16 + (lane & 15)][(j + z) * 16 + (lane >> 4) * 8]));
#pragma unroll
          for (int z = 0; z < 4; ++z) mma2(st_acc[2 * (j + z)], st_acc[2 * (j + z) + 1], big, x[z]);
#pragma unroll
          for (int z = 0; z < 4; ++z) mma2(st_acc[2 * (j + z)], st_acc[2 * (j + z) + 1], rest, x[z]);
        }
      }
    }
    if constexpr (MODE == MEMORY) {
      // the outputs' denominators; then the normaliser moves on (a thread per channel, read again in the next chunk only)
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int z = 0; z < 2; ++z) {
          const int i = j * 8 + t2 + z;
          float den = sm.x2[i] * sm.x4[i];
#pragma unroll
          for (int b = 0; b <= j / 2; ++b) den += sm.part[i][b];
          den = __fdividef(1.f, fmaxf(fabsf(den), sm.x3[i]) + 1e-6f);
          acc[j][z] *= den;
          acc[j][z + 2] *= den;
        }
      constexpr int PARTS = CTHREADS / DK;         // a part takes every PARTS-th token
      float s = sm.n[tid] * keep;
#pragma unroll 8
      for (int j = tid / DK; j < n; j += PARTS) s += sm.x5[j] * __bfloat162float(sk_[j][tid % DK]);
      sm.n[tid] = s;
      m = sm.end[1];
    }
    // ---- outputs: this warp's columns of the value tile hold them for wide stores (no other warp reads those columns)
    __syncwarp();
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) sv_[j * 8 + t2 + (e & 1)][w0 + lg + (e >> 1) * 8] = __float2bfloat16(acc[j][e]);
    __syncwarp();
#pragma unroll
    for (int i = lane; i < CT * 2; i += 32) {
      const int t = i >> 1, c = w0 + (i & 1) * 8;
      if (t < n && c < vcols) *reinterpret_cast<uint4*>(o + (t0 + t) * o_stride + c) = *reinterpret_cast<const uint4*>(&sv_[t][c]);
    }
  }
  if (S != nullptr && len > 0) {
#pragma unroll
    for (int n = 0; n < NK; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int kr = n * 8 + t2 + (e & 1), vc = c0 + w0 + lg + (e >> 1) * 8;
        if (kr < dk && vc < dv) S[static_cast<long long>(kr) * dv + vc] = st_acc[n][e];
      }
    if (MODE == MEMORY && blockIdx.y == 0) {
      __syncthreads();
      if (tid < dk) {
        float s = 0.f;
#pragma unroll
        for (int x = 0; x < CTHREADS / DK; ++x) s += sm.n[x * DK + tid];
        p.n[rh * dk + tid] = s;
      }
      if (tid == 0) p.m[rh] = m;
    }
  }
  for (int i = tid; i < (S_len - len) * (VT / 8); i += CTHREADS) {
    const int t = len + i / (VT / 8), c = (i % (VT / 8)) * 8;
    if (c < vcols) *reinterpret_cast<uint4*>(o + t * o_stride + c) = make_uint4(0, 0, 0, 0);
  }
}

// ---------------------------------------------------------------------------------------------------------------- wkv
constexpr int WT = 16, VT = 64, CTHREADS = 128;             // tokens per chunk; value columns and threads of a block

template <int DK>
struct WkvSmem {
  bf16 q[WT][DK + 8], k[WT][DK + 8], v[WT][VT + 8];
  bf16 qs[2][WT][DK + 8], ks[2][WT][DK + 8];       // q e^(L of the token before), k e^(L_end - L): value, rest
  bf16 p[2][WT][WT + 8];
  float L[WT + 1][DK + 4];                         // sums of the log decays; row 0 is zero
  float keep[DK], u[DK];
};

// grid (H, ceil(dv / VT), rows)
template <int DK>
__global__ void __launch_bounds__(CTHREADS)
wkv_chunks_kernel(Args<bf16> p) {
  extern __shared__ __align__(16) uint8_t raw[];
  WkvSmem<DK>& sm = *reinterpret_cast<WkvSmem<DK>*>(raw);
  constexpr int NK = DK / 8;
  const int dk = p.dk, dv = p.dv, S_len = p.S, h = blockIdx.x, row = blockIdx.z, c0 = blockIdx.y * VT;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, lg = lane >> 2, t2 = (lane & 3) * 2;
  const long long t_row = static_cast<long long>(row) * S_len;
  const int first = p.positions[t_row], len = first < 0 ? 0 : min(p.lengths[row] - first, S_len);
  const int r = p.row_ids == nullptr ? row : p.row_ids[row];
  const long long rh = static_cast<long long>(r) * p.H + h;
  const bf16 *qb = p.q + t_row * p.q_stride + h * dk, *kb = p.k + t_row * p.k_stride + h * dk, *vb = p.v + t_row * p.v_stride + h * dv + c0;
  const float* lb = p.log_decay + (t_row * p.H + h) * dk;
  const long long l_stride = static_cast<long long>(p.H) * dk, o_stride = static_cast<long long>(p.H) * dv;
  bf16* o = p.out + (t_row * p.H + h) * dv + c0;
  float* S = p.state == nullptr ? nullptr : p.state + rh * dk * dv;
  const bool held = S != nullptr && first > 0;
  const int w0 = warp * 16, vcols = min(VT, dv - c0);
  float st_acc[NK][4];
#pragma unroll
  for (int n = 0; n < NK; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int kr = n * 8 + t2 + (e & 1), vc = c0 + w0 + lg + (e >> 1) * 8;
      st_acc[n][e] = held && kr < dk && vc < dv ? S[static_cast<long long>(kr) * dv + vc] : 0.f;
    }
  for (int c = tid; c < DK; c += CTHREADS) {
    sm.u[c] = c < dk ? ld(p.u + h * dk + c) : 0.f;
    sm.L[0][c] = 0.f;
  }
  int my_i = 1;                                    // this thread's pair of tokens
  while (my_i < WT - 1 && my_i * (my_i + 1) / 2 <= tid) ++my_i;
  const int my_j = tid - my_i * (my_i - 1) / 2;
  // the next chunk's rows wait in registers
  constexpr int QV = WT * DK / 8 / CTHREADS > 0 ? WT * DK / 8 / CTHREADS : 1, LV = WT * DK / 4 / CTHREADS;
  uint4 rq[QV], rk[QV], rv;
  float4 rl[LV];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < QV; ++i) {
      const int x = tid + i * CTHREADS, t = x / (DK / 8), c = (x % (DK / 8)) * 8;
      const bool ok = t0 + t < len && c < dk;
      rq[i] = row16(qb + (t0 + t) * p.q_stride + c, ok);
      rk[i] = row16(kb + (t0 + t) * p.k_stride + c, ok);
    }
    {
      const int t = tid / (VT / 8), c = (tid % (VT / 8)) * 8;
      rv = row16(vb + (t0 + t) * p.v_stride + c, t0 + t < len && c < vcols);
    }
#pragma unroll
    for (int i = 0; i < LV; ++i) {                 // tokens past the end decay nothing
      const int x = tid + i * CTHREADS, t = x / (DK / 4), c = (x % (DK / 4)) * 4;
      rl[i] = t0 + t < len && c < dk ? *reinterpret_cast<const float4*>(lb + (t0 + t) * l_stride + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  if (len > 0) fetch(0);
  for (int t0 = 0; t0 < len; t0 += WT) {
    const int n = min(WT, len - t0);
    __syncthreads();                               // the chunk before has been read
#pragma unroll
    for (int i = 0; i < QV; ++i) {
      const int x = tid + i * CTHREADS, t = x / (DK / 8), c = (x % (DK / 8)) * 8;
      *reinterpret_cast<uint4*>(&sm.q[t][c]) = rq[i];
      *reinterpret_cast<uint4*>(&sm.k[t][c]) = rk[i];
    }
    *reinterpret_cast<uint4*>(&sm.v[tid / (VT / 8)][(tid % (VT / 8)) * 8]) = rv;
#pragma unroll
    for (int i = 0; i < LV; ++i) {
      const int x = tid + i * CTHREADS, t = x / (DK / 4), c = (x % (DK / 4)) * 4;
      *reinterpret_cast<float4*>(&sm.L[t + 1][c]) = rl[i];
    }
    __syncthreads();
    if (t0 + WT < len) fetch(t0 + WT);
    for (int c = tid; c < DK; c += CTHREADS) {
      float s = 0.f;
#pragma unroll
      for (int t = 1; t <= WT; ++t) { s += sm.L[t][c]; sm.L[t][c] = s; }
      sm.keep[c] = expf(s);
    }
    __syncthreads();
    // ---- q and k with their decays, and the scores of the token pairs
    for (int i = tid; i < WT * (DK / 2); i += CTHREADS) {
      const int t = i / (DK / 2), c = (i % (DK / 2)) * 2;
      const uint32_t qq = *reinterpret_cast<const uint32_t*>(&sm.q[t][c]), kk = *reinterpret_cast<const uint32_t*>(&sm.k[t][c]);
      const float2 a = *reinterpret_cast<const float2*>(&sm.L[t][c]), b = *reinterpret_cast<const float2*>(&sm.L[t + 1][c]),
                   e = *reinterpret_cast<const float2*>(&sm.L[WT][c]);
      uint32_t big, rest;
      split2(lo_f(qq) * __expf(a.x), hi_f(qq) * __expf(a.y), big, rest);
      *reinterpret_cast<uint32_t*>(&sm.qs[0][t][c]) = big;
      *reinterpret_cast<uint32_t*>(&sm.qs[1][t][c]) = rest;
      split2(lo_f(kk) * __expf(e.x - b.x), hi_f(kk) * __expf(e.y - b.y), big, rest);
      *reinterpret_cast<uint32_t*>(&sm.ks[0][t][c]) = big;
      *reinterpret_cast<uint32_t*>(&sm.ks[1][t][c]) = rest;
    }
    auto score = [&](int i, int j, float s) {
      const bf16 big = __float2bfloat16(s);
      sm.p[0][i][j] = big;
      sm.p[1][i][j] = __float2bfloat16(s - __bfloat162float(big));
    };
    if (tid < WT * (WT - 1) / 2) {                 // a pair below the diagonal per thread
      const int i = my_i, j = my_j;
      float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
      for (int c = 0; c < DK; c += 4) {
        const uint2 qq = *reinterpret_cast<const uint2*>(&sm.q[i][c]), kk = *reinterpret_cast<const uint2*>(&sm.k[j][c]);
        const float4 a = *reinterpret_cast<const float4*>(&sm.L[i][c]), b = *reinterpret_cast<const float4*>(&sm.L[j + 1][c]);
        s[0] += lo_f(qq.x) * lo_f(kk.x) * __expf(a.x - b.x);
        s[1] += hi_f(qq.x) * hi_f(kk.x) * __expf(a.y - b.y);
        s[2] += lo_f(qq.y) * lo_f(kk.y) * __expf(a.z - b.z);
        s[3] += hi_f(qq.y) * hi_f(kk.y) * __expf(a.w - b.w);
      }
      score(i, j, (s[0] + s[1]) + (s[2] + s[3]));
      sm.p[0][j][i] = sm.p[1][j][i] = __float2bfloat16(0.f);
    }
    {                                              // the token itself: eight threads each
      const int i = tid >> 3;
      float s = 0.f;
#pragma unroll
      for (int c = (tid & 7) * 2; c < DK; c += 16) {
        const uint32_t qq = *reinterpret_cast<const uint32_t*>(&sm.q[i][c]), kk = *reinterpret_cast<const uint32_t*>(&sm.k[i][c]);
        s += lo_f(qq) * lo_f(kk) * sm.u[c] + hi_f(qq) * hi_f(kk) * sm.u[c + 1];
      }
#pragma unroll
      for (int q = 4; q > 0; q >>= 1) s += __shfl_xor_sync(0xffffffffu, s, q);
      if ((tid & 7) == 0) score(i, i, s);
    }
    __syncthreads();
    // ---- outputs [16 values, 16 tokens]
    float acc[2][4] = {}, acc1[2][4] = {}, acc2[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t big[4], rest[4], x[4], y[4];
      as_operand(st_acc[kk / 8], st_acc[kk / 8 + 1], big, rest);
      ldsm4(x, smem_addr(&sm.qs[0][(lane & 7) + (lane >> 4) * 8][kk + ((lane >> 3) & 1) * 8]));
      ldsm4(y, smem_addr(&sm.qs[1][(lane & 7) + (lane >> 4) * 8][kk + ((lane >> 3) & 1) * 8]));
      mma2(acc[0], acc[1], big, x);
      mma2(acc1[0], acc1[1], rest, x);
      mma2(acc2[0], acc2[1], big, y);
    }
    uint32_t vt[4], x[4], y[4];
    ldsm4_t(vt, smem_addr(&sm.v[(lane & 7) + (lane >> 4) * 8][w0 + ((lane >> 3) & 1) * 8]));
    ldsm4(x, smem_addr(&sm.p[0][(lane & 7) + (lane >> 4) * 8][((lane >> 3) & 1) * 8]));
    ldsm4(y, smem_addr(&sm.p[1][(lane & 7) + (lane >> 4) * 8][((lane >> 3) & 1) * 8]));
    mma2(acc[0], acc[1], vt, x);
    mma2(acc1[0], acc1[1], vt, y);
#pragma unroll
    for (int z = 0; z < 2; ++z)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[z][e] += acc1[z][e] + acc2[z][e];
    // ---- the state after the chunk
#pragma unroll
    for (int j = 0; j < NK; ++j) {
      const float2 w = *reinterpret_cast<const float2*>(&sm.keep[j * 8 + t2]);
      st_acc[j][0] *= w.x; st_acc[j][1] *= w.y; st_acc[j][2] *= w.x; st_acc[j][3] *= w.y;
    }
#pragma unroll
    for (int part = 0; part < 2; ++part)
#pragma unroll
      for (int j = 0; j < NK / 2; ++j) {
        ldsm4_t(x, smem_addr(&sm.ks[part][lane & 15][j * 16 + (lane >> 4) * 8]));
        mma2(st_acc[2 * j], st_acc[2 * j + 1], vt, x);
      }
    __syncwarp();
#pragma unroll
    for (int z = 0; z < 2; ++z)
#pragma unroll
      for (int e = 0; e < 4; ++e) sm.v[z * 8 + t2 + (e & 1)][w0 + lg + (e >> 1) * 8] = __float2bfloat16(acc[z][e]);
    __syncwarp();
    {
      const int t = lane >> 1, c = w0 + (lane & 1) * 8;
      if (t < n && c < vcols) *reinterpret_cast<uint4*>(o + (t0 + t) * o_stride + c) = *reinterpret_cast<const uint4*>(&sm.v[t][c]);
    }
  }
  if (S != nullptr && len > 0) {
#pragma unroll
    for (int n = 0; n < NK; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int kr = n * 8 + t2 + (e & 1), vc = c0 + w0 + lg + (e >> 1) * 8;
        if (kr < dk && vc < dv) S[static_cast<long long>(kr) * dv + vc] = st_acc[n][e];
      }
  }
  for (int i = tid; i < (S_len - len) * (VT / 8); i += CTHREADS) {
    const int t = len + i / (VT / 8), c = (i % (VT / 8)) * 8;
    if (c < vcols) *reinterpret_cast<uint4*>(o + t * o_stride + c) = make_uint4(0, 0, 0, 0);
  }
}

template <typename K>
int chunks_go(K kernel, size_t smem, int columns, const Args<bf16>& p, cudaStream_t stream) {
  if (smem > 225 * 1024) return -3;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kernel<<<dim3(p.H, (p.dv + columns - 1) / columns, p.R), columns * 2, smem, stream>>>(p);
  return static_cast<int>(cudaGetLastError());
}

template <int MODE, int DK>
int chunks_of(const Args<bf16>& p, cudaStream_t stream) {
  // wide blocks form a head's scores once instead of twice; narrow ones pay while both halves find an SM each
  constexpr long long HALF_THE_SMS = 74;
  if (p.dv > 64 && static_cast<long long>(p.R) * p.H * ((p.dv + 127) / 128) > HALF_THE_SMS)
    return chunks_go(gated_chunks_kernel<MODE, DK, 8>, sizeof(ChunkSmem<MODE, DK, 8>), 128, p, stream);
  return chunks_go(gated_chunks_kernel<MODE, DK, 4>, sizeof(ChunkSmem<MODE, DK, 4>), 64, p, stream);
}

}  // namespace gated
}  // namespace dewb

using namespace dewb::gated;

// The chunked tensor-core form: bf16; dk, dv and the strides multiples of 8, dk at most 128; q, k, v, out (and log_decay) on 16-byte boundaries.
extern "C" int dewb_gated_chunks(int mode, const dewb_gated_args* a, void* stream_ptr) {
  if (a == nullptr) return -3;
  if (a->R <= 0 || a->S <= 0) return 0;
  if (!args_ok(mode, *a) || a->dk % 8 || a->dv % 8 || a->dk > 128 || a->q_stride % 8 || a->k_stride % 8 || a->v_stride % 8) return -3;
  if (!dewb::rows::aligned(a->q, 16) || !dewb::rows::aligned(a->k, 16) || !dewb::rows::aligned(a->v, 16) || !dewb::rows::aligned(a->out, 16) ||
      !dewb::rows::aligned(a->log_decay, 16) || (a->dv + 63) / 64 > 65535 || (mode == MEMORY && a->state != nullptr && a->n_before == nullptr))
    return -3;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_ptr);
  const Args<bf16> p(*a);
  const bool wide = p.dk > 64;
  if (mode == WKV) return wide ? chunks_go(wkv_chunks_kernel<128>, sizeof(WkvSmem<128>), VT, p, stream) : chunks_go(wkv_chunks_kernel<64>, sizeof(WkvSmem<64>), VT, p, stream);
  if (mode == MEMORY) return wide ? chunks_of<MEMORY, 128>(p, stream) : chunks_of<MEMORY, 64>(p, stream);
  return wide ? chunks_of<DELTA, 128>(p, stream) : chunks_of<DELTA, 64>(p, stream);
}
