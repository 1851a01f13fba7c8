// Prompt form of the SSD recurrence on tensor cores (bf16 activations, fp32 state); operands from sx_ssd_operands.
//
// One CTA walks one portion for one head and up to 64 of its value columns in chunks of 64 tokens. With cs_t the running sum
// of the logarithms of the decays in the chunk and S0 the state in front of it,
//   y_t = exp(cs_t) S0^T C_t + sum_{s <= t} M_ts x_s,    M_ts = (C_t . B_s) exp(cs_t - cs_s) dt_s
//   S   = exp(cs_last) S0 + sum_s B_s (exp(cs_last - cs_s) dt_s x_s)^T
// All products are mma.sync m16n8k16 with the transposed state S^T [columns, N] as an operand or result: a warp owns 16 value
// columns, and the accumulator fragments of its S^T are read back as A fragments, so the state never leaves registers. x, B
// and C are bf16 as the convolution rounds them; an fp32 factor (the state in the read-out, the weighted x in the update) is
// split in two bf16 terms, which keeps 16 bits of every product's factor and fp32 sums. M is rounded once, like the
// probabilities of an attention. Rows past a portion's end are zero.
#include "tc_common.cuh"
#include "ragged.cuh"
#include "sx_api.h"

namespace sx {

constexpr int SS_Q = 64;               // tokens per chunk
constexpr int SS_LX = 64 + 8;          // row pitches (bf16 entries)

struct SsdScanParams {
  SxSsdArgs a;
  RaggedView rv;
};

template <int KN>      // steps of 16 state rows
struct SsdScanCfg {
  static constexpr int LN = KN * 16 + 8;
  static constexpr int STAGE = SS_Q * (SS_LX + 2 * LN);          // x, B, C
  static constexpr int OFF_Z = 2 * STAGE, OFF_M = OFF_Z + SS_Q * SS_LX;
  static constexpr int OFF_V = OFF_M + SS_Q * SS_LX;             // per warp: cs [64], dt [64] (fp32)
  static constexpr int SMEM = OFF_V * 2 + 4 * 2 * SS_Q * 4;
  static_assert(SMEM <= 227 * 1024, "shared memory");
};

__device__ __forceinline__ void ss_cp16(uint32_t dst, const void* src, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ss_ldsm4(uint32_t (&r)[4], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(p) : "memory");
}
__device__ __forceinline__ void ss_ldsm4t(uint32_t (&r)[4], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(p) : "memory");
}
__device__ __forceinline__ void ss_stsm4t(uint32_t p, uint32_t a, uint32_t b, uint32_t c, uint32_t d) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};" ::"r"(p), "r"(a), "r"(b), "r"(c), "r"(d) : "memory");
}
__device__ __forceinline__ void ss_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float lo_f(uint32_t p) { return __uint_as_float(p << 16); }
__device__ __forceinline__ float hi_f(uint32_t p) { return __uint_as_float(p & 0xffff0000u); }
// (x, y) in two packed bf16 terms
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - lo_f(hi), y - hi_f(hi));
}

template <int KN>
__global__ void __launch_bounds__(128, KN <= 8 ? 2 : 1) ssd_scan_kernel(const SsdScanParams P) {
  using Cfg = SsdScanCfg<KN>;
  using bf = __nv_bfloat16;
  extern __shared__ __align__(128) uint8_t smem[];
  const SxSsdArgs& p = P.a;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, seq = blockIdx.z, grp = h / (p.H / p.G), c0 = blockIdx.x * 64 + warp * 16;   // first column of this warp
  const int row0 = P.rv.cu[seq], len = P.rv.cu[seq + 1] - row0;
  if (len <= 0) return;
  const int n_ch = (len + SS_Q - 1) / SS_Q, ksteps = (p.N + 15) / 16;
  bf* sm = reinterpret_cast<bf*>(smem);
  bf* sZ = sm + Cfg::OFF_Z;
  float* s_cs = reinterpret_cast<float*>(smem + Cfg::OFF_V * 2) + warp * 2 * SS_Q;
  float* s_dt = s_cs + SS_Q;
  const uint32_t a_sm = smem_u32(smem), a_z = smem_u32(sZ), a_m = a_sm + Cfg::OFF_M * 2;
  const bf* X = reinterpret_cast<const bf*>(p.x) + (long long)row0 * p.H * p.xp + h * p.xp;
  const bf* B = reinterpret_cast<const bf*>(p.b) + ((long long)row0 * p.G + grp) * p.np;
  const bf* Cc = reinterpret_cast<const bf*>(p.c) + ((long long)row0 * p.G + grp) * p.np;
  const bf* Z = reinterpret_cast<const bf*>(p.u) + (long long)row0 * p.u_ld + (long long)h * p.P;
  bf* Y = reinterpret_cast<bf*>(p.y) + (long long)row0 * p.y_ld + (long long)h * p.P;
  const bool z_vec = p.P % 8 == 0 && p.u_ld % 8 == 0 && (reinterpret_cast<uintptr_t>(p.u) & 15) == 0;
  const bool y_vec = p.P % 8 == 0 && p.y_ld % 8 == 0 && (reinterpret_cast<uintptr_t>(p.y) & 15) == 0;

  // x columns of a warp are loaded (and read) by that warp only; B and C by all
  auto load = [&](int ci) {
    if (ci < n_ch) {
      const int t0 = ci * SS_Q;
      const uint32_t st = a_sm + (ci & 1) * Cfg::STAGE * 2;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = i * 16 + (lane >> 1), c = c0 + (lane & 1) * 8;
        const bool ok = t0 + r < len && c < p.xp;
        ss_cp16(st + (r * SS_LX + warp * 16 + (lane & 1) * 8) * 2, ok ? X + (long long)(t0 + r) * p.H * p.xp + c : X, ok);
      }
      constexpr int PR = KN * 2;            // 16-byte pieces of a row
#pragma unroll
      for (int i = 0; i < SS_Q * PR / 128; ++i) {
        const int idx = i * 128 + tid, r = idx / PR, c = (idx % PR) * 8;
        const bool ok = t0 + r < len && c < p.np;
        const long long off = ok ? (long long)(t0 + r) * p.G * p.np + c : 0;
        ss_cp16(st + (SS_Q * SS_LX + r * Cfg::LN + c) * 2, B + off, ok);
        ss_cp16(st + (SS_Q * (SS_LX + Cfg::LN) + r * Cfg::LN + c) * 2, Cc + off, ok);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_z = [&](int t0) {
    if (z_vec) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = i * 16 + (lane >> 1), c = c0 + (lane & 1) * 8;
        const bool ok = t0 + r < len && c < p.P;
        ss_cp16(a_z + (r * SS_LX + warp * 16 + (lane & 1) * 8) * 2, ok ? Z + (long long)(t0 + r) * p.u_ld + c : Z, ok);
      }
    } else {
      for (int i = lane; i < SS_Q * 16; i += 32) {
        const int r = i >> 4, c = c0 + (i & 15);
        sZ[r * SS_LX + warp * 16 + (i & 15)] = t0 + r < len && c < p.P ? Z[(long long)(t0 + r) * p.u_ld + c] : __float2bfloat16_rn(0.f);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // step sizes and decays of a chunk: two neighbouring tokens per lane
  float nla[2], ndt[2];
  auto load_steps = [&](int t0) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = t0 + 2 * lane + e;
      const long long o = (long long)(row0 + t) * p.H + h;
      nla[e] = t < len ? p.la[o] : 0.f;
      ndt[e] = t < len ? p.dt[o] : 0.f;
    }
  };
  load(0);
  load_steps(0);
  // transposed state: row c0 + g + 8 (e >> 1), state row 8 j + 2 t4 + (e & 1)
  float S[2 * KN][4];
  float* st = p.state + ((long long)P.rv.slot[seq] * p.H + h) * p.N * p.P;
  const bool fresh = P.rv.pos0[seq] == 0;
#pragma unroll
  for (int j = 0; j < 2 * KN; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 8 * j + 2 * t4 + (e & 1), c = c0 + g + (e >> 1) * 8;
      S[j][e] = !fresh && n < p.N && c < p.P ? st[(long long)n * p.P + c] : 0.f;
    }
  const float D = p.D[h];
  // lane parts of the ldmatrix addresses: rows of a 16 x 16 tile whose quarters go (row 0, col 0), (0, 8), (8, 0), (8, 8) or
  // (0, 0), (8, 0), (0, 8), (8, 8)
  const int rc_r = (lane & 7) + (lane >> 4) * 8, rc_c = ((lane >> 3) & 1) * 8;
  const int cr_r = lane & 15, cr_c = (lane >> 4) * 8;

  for (int ci = 0; ci < n_ch; ++ci) {
    const int t0 = ci * SS_Q;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();             // the chunk is there, and everybody has left the previous one
    const uint32_t sx_ = a_sm + (ci & 1) * Cfg::STAGE * 2, sb_ = sx_ + SS_Q * SS_LX * 2, sc_ = sb_ + SS_Q * Cfg::LN * 2;
    float total;
    {
      float a = nla[0] + nla[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, a, o);
        if (lane >= o) a += v;
      }
      *reinterpret_cast<float2*>(s_cs + 2 * lane) = make_float2(a - nla[1], a);
      *reinterpret_cast<float2*>(s_dt + 2 * lane) = make_float2(ndt[0], ndt[1]);
      total = __shfl_sync(0xffffffffu, a, 31);
      __syncwarp();
    }
    load_z(t0);
    load(ci + 1);
    load_steps(t0 + SS_Q);
    // M, rows 16 warp .. 16 warp + 15
    {
      float G[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < KN; ++kk) {
        if (kk >= ksteps) break;
        uint32_t a[4];
        ss_ldsm4(a, sc_ + ((warp * 16 + cr_r) * Cfg::LN + kk * 16 + cr_c) * 2);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (i > warp) break;
          uint32_t b[4];
          ss_ldsm4(b, sb_ + ((i * 16 + rc_r) * Cfg::LN + kk * 16 + rc_c) * 2);
          ss_mma(G[2 * i], a, b[0], b[1]);
          ss_mma(G[2 * i + 1], a, b[2], b[3]);
        }
      }
      const float ct[2] = {s_cs[warp * 16 + g], s_cs[warp * 16 + g + 8]};
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (i > 2 * warp + 1) break;
        const int s = i * 8 + t4 * 2;
        const float2 cs = *reinterpret_cast<const float2*>(s_cs + s), dt = *reinterpret_cast<const float2*>(s_dt + s);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = warp * 16 + g + 8 * r;
          const float m0 = s <= t ? G[i][2 * r] * __expf(ct[r] - cs.x) * dt.x : 0.f;
          const float m1 = s + 1 <= t ? G[i][2 * r + 1] * __expf(ct[r] - cs.y) * dt.y : 0.f;
          asm volatile("st.shared.b32 [%0], %1;" ::"r"(a_m + (t * SS_LX + s) * 2), "r"(pack_bf16x2(m0, m1)) : "memory");
        }
      }
    }
    // what the state in front of the chunk contributes: O^T = S^T C^T, columns scaled by exp(cs)
    float O[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) O[i][0] = O[i][1] = O[i][2] = O[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < KN; ++kk) {
      if (kk >= ksteps) break;
      uint32_t ah[4], al[4];
      split2(S[2 * kk][0], S[2 * kk][1], ah[0], al[0]);
      split2(S[2 * kk][2], S[2 * kk][3], ah[1], al[1]);
      split2(S[2 * kk + 1][0], S[2 * kk + 1][1], ah[2], al[2]);
      split2(S[2 * kk + 1][2], S[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        uint32_t b[4];
        ss_ldsm4(b, sc_ + ((i * 16 + rc_r) * Cfg::LN + kk * 16 + rc_c) * 2);
        ss_mma(O[2 * i], al, b[0], b[1]);
        ss_mma(O[2 * i + 1], al, b[2], b[3]);
        ss_mma(O[2 * i], ah, b[0], b[1]);
        ss_mma(O[2 * i + 1], ah, b[2], b[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float2 cs = *reinterpret_cast<const float2*>(s_cs + i * 8 + t4 * 2);
      const float e0 = __expf(cs.x), e1 = __expf(cs.y);
      O[i][0] *= e0; O[i][1] *= e1; O[i][2] *= e0; O[i][3] *= e1;
    }
    // x^T fragments: columns g (+ 8), tokens 16 kk + 2 t4 (+ 1) and 8 further
    uint32_t x[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) ss_ldsm4t(x[kk], sx_ + ((kk * 16 + rc_r) * SS_LX + warp * 16 + rc_c) * 2);
    __syncthreads();             // M is complete
    // what the chunk's own tokens contribute: O^T += x^T M^T
#pragma unroll
    for (int kk = 0; kk < 4; ++kk)
#pragma unroll
      for (int i = kk; i < 4; ++i) {
        uint32_t b[4];
        ss_ldsm4(b, a_m + ((i * 16 + rc_r) * SS_LX + kk * 16 + rc_c) * 2);
        ss_mma(O[2 * i], x[kk], b[0], b[1]);
        ss_mma(O[2 * i + 1], x[kk], b[2], b[3]);
      }
    // state behind the chunk
    {
      const float f = __expf(total);
#pragma unroll
      for (int j = 0; j < 2 * KN; ++j) {
        S[j][0] *= f; S[j][1] *= f; S[j][2] *= f; S[j][3] *= f;
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t ah[4], al[4];
#pragma unroll
      for (int e = 0; e < 2; ++e) {          // tokens 16 kk + 8 e + 2 t4 and the next
        const int s = kk * 16 + 8 * e + t4 * 2;
        const float2 cs = *reinterpret_cast<const float2*>(s_cs + s), dt = *reinterpret_cast<const float2*>(s_dt + s);
        const float w0 = __expf(total - cs.x) * dt.x, w1 = __expf(total - cs.y) * dt.y;
        split2(lo_f(x[kk][2 * e]) * w0, hi_f(x[kk][2 * e]) * w1, ah[2 * e], al[2 * e]);
        split2(lo_f(x[kk][2 * e + 1]) * w0, hi_f(x[kk][2 * e + 1]) * w1, ah[2 * e + 1], al[2 * e + 1]);
      }
#pragma unroll
      for (int j = 0; j < KN; ++j) {
        if (j >= ksteps) break;
        uint32_t b[4];
        ss_ldsm4t(b, sb_ + ((kk * 16 + cr_r) * Cfg::LN + j * 16 + cr_c) * 2);
        ss_mma(S[2 * j], al, b[0], b[1]);
        ss_mma(S[2 * j + 1], al, b[2], b[3]);
        ss_mma(S[2 * j], ah, b[0], b[1]);
        ss_mma(S[2 * j + 1], ah, b[2], b[3]);
      }
    }
    // skip connection and output gate in the fragment layout, then through this warp's own x columns to rows
    asm volatile("cp.async.wait_group 1;" ::: "memory");      // z; the next chunk may still be on its way
    __syncwarp();
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t z[4], y[4];
      ss_ldsm4t(z, a_z + ((kk * 16 + rc_r) * SS_LX + warp * 16 + rc_c) * 2);
#pragma unroll
      for (int i = 0; i < 4; ++i) {          // i = 2 (token half) + (column half)
        const float o0 = fmaf(D, lo_f(x[kk][i]), O[2 * kk + (i >> 1)][2 * (i & 1)]);
        const float o1 = fmaf(D, hi_f(x[kk][i]), O[2 * kk + (i >> 1)][2 * (i & 1) + 1]);
        y[i] = pack_bf16x2(o0 * silu_act<bf>(lo_f(z[i])), o1 * silu_act<bf>(hi_f(z[i])));
      }
      ss_stsm4t(sx_ + ((kk * 16 + rc_r) * SS_LX + warp * 16 + rc_c) * 2, y[0], y[1], y[2], y[3]);
    }
    __syncwarp();
    const bf* sx_p = sm + (ci & 1) * Cfg::STAGE + warp * 16;
    if (y_vec) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = i * 16 + (lane >> 1), c = (lane & 1) * 8;
        if (t0 + r < len && c0 + c < p.P)
          *reinterpret_cast<uint4*>(Y + (long long)(t0 + r) * p.y_ld + c0 + c) = *reinterpret_cast<const uint4*>(sx_p + r * SS_LX + c);
      }
    } else {
      for (int i = lane; i < SS_Q * 16; i += 32) {
        const int r = i >> 4, c = i & 15;
        if (t0 + r < len && c0 + c < p.P) Y[(long long)(t0 + r) * p.y_ld + c0 + c] = sx_p[r * SS_LX + c];
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 2 * KN; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 8 * j + 2 * t4 + (e & 1), c = c0 + g + (e >> 1) * 8;
      if (n < p.N && c < p.P) st[(long long)n * p.P + c] = S[j][e];
    }
}

template <int KN>
static int launch_ssd_scan(const SsdScanParams& p, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(ssd_scan_kernel<KN>, cudaFuncAttributeMaxDynamicSharedMemorySize, SsdScanCfg<KN>::SMEM) != cudaSuccess) return -10;
    set = true;
  }
  ssd_scan_kernel<KN><<<dim3((p.a.P + 63) / 64, p.a.H, p.rv.n), 128, SsdScanCfg<KN>::SMEM, st>>>(p);
  return last_rc();
}

}  // namespace sx
using namespace sx;

// 1 when sx_ssd_scan takes these sizes.
extern "C" int sx_ssd_scan_ok(int P, int N) { return P > 0 && N > 0 && N <= 256; }

extern "C" int sx_ssd_scan(const SxSsdArgs* a, cudaStream_t st) {
  if (a->ragged.n <= 0) return 0;
  if (!sx_ssd_scan_ok(a->P, a->N) || a->f32 || a->G <= 0 || a->H % a->G || a->xp % 8 || a->np % 8 || a->xp < a->P || a->np < a->N ||
      a->H > 65535 || a->ragged.n > 65535)
    return -1;
  if ((reinterpret_cast<uintptr_t>(a->x) | reinterpret_cast<uintptr_t>(a->b) | reinterpret_cast<uintptr_t>(a->c)) & 15) return -3;
  const SsdScanParams p{*a, view(&a->ragged)};
  if (a->N <= 32) return launch_ssd_scan<2>(p, st);
  if (a->N <= 64) return launch_ssd_scan<4>(p, st);
  if (a->N <= 128) return launch_ssd_scan<8>(p, st);
  return launch_ssd_scan<16>(p, st);
}
