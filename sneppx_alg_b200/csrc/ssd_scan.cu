// Prompt form of the SSD recurrence on tensor cores (bf16 activations, fp32 state); operands from sx_ssd_operands.
//
// One CTA of eight warps walks one portion for one head and up to 64 of its value columns in chunks of 64 tokens. With cs_t the running sum
// of the logarithms of the decays in the chunk and S0 the state in front of it,
//   y_t = exp(cs_t) S0^T C_t + sum_{s <= t} M_ts x_s,    M_ts = (C_t . B_s) exp(cs_t - cs_s) dt_s
//   S   = exp(cs_last) S0 + sum_s B_s (exp(cs_last - cs_s) dt_s x_s)^T
// All products are mma.sync m16n8k16 with the transposed state S^T [columns, N] as an operand or result: a warp owns 16 value
// columns of one half of N, and the accumulator fragments of its S^T are read back as A fragments, so the state never leaves
// registers. The two warps of a column tile exchange their halves' read-outs through shared memory and finish two of the four
// 16-token blocks each (first and last, second and third: equal work under the triangle). x, B
// and C are bf16 as the convolution rounds them; an fp32 factor (the state in the read-out, the weighted x in the update) is
// split in two bf16 terms, which keeps 16 bits of every product's factor and fp32 sums. M is rounded once, like the
// probabilities of an attention. Rows past a portion's end are zero.
//
// With few sequences their portions are cut into segments that run side by side: a first pass (STATE) walks every segment but
// a sequence's last from an empty state and keeps only what it leaves, a second chains these from the stored state to the
// state in front of every segment, and the full pass starts from there.
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
  static constexpr int STAGE = SS_Q * (SS_LX + LN);              // x, B (two stages)
  static constexpr int OFF_C = 2 * STAGE, OFF_Z = OFF_C + SS_Q * LN, OFF_M = OFF_Z + SS_Q * SS_LX, OFF_V = OFF_M + SS_Q * SS_LX;
  static constexpr int OFF_X = OFF_V * 2 + 8 * 4 * SS_Q * 4;     // bytes from here: after per warp cs, dt, exp(cs), weights of the update [64 each]
  static constexpr int SMEM = OFF_X + 2 * 4 * 4 * 32 * 16;       // exchange: [receiving half][column tile][4 tiles][lane] float4
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
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float lo_f(uint32_t p) { return __uint_as_float(p << 16); }
__device__ __forceinline__ float hi_f(uint32_t p) { return __uint_as_float(p & 0xffff0000u); }
// (x, y) in two packed bf16 terms
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - lo_f(hi), y - hi_f(hi));
}

template <int KN, bool STATE>
__global__ void __launch_bounds__(256, KN <= 8 ? 2 : 1) ssd_scan_kernel(const SsdScanParams P) {
  using Cfg = SsdScanCfg<KN>;
  using bf = __nv_bfloat16;
  constexpr int KH = KN / 2;           // k steps of a half
  extern __shared__ __align__(128) uint8_t smem[];
  const SxSsdArgs& p = P.a;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int pw = warp & 3, half = warp >> 2;                     // column tile, half of N
  const int h = blockIdx.y, z_id = blockIdx.z, grp = h / (p.H / p.G), c0 = blockIdx.x * 64 + pw * 16;   // first column of this warp
  const int seq = p.n_seg ? p.seg_seq[z_id] : z_id, off = p.n_seg ? (z_id - p.seg_first[seq]) * p.seg_rows : 0;
  const int row0 = P.rv.cu[seq] + off, left = P.rv.cu[seq + 1] - row0, len = p.n_seg ? min(left, p.seg_rows) : left;
  const bool last = len == left;       // the sequence's last (or only) segment
  if (len <= 0 || (STATE && last)) return;
  const int n_ch = (len + SS_Q - 1) / SS_Q, ksteps = (p.N + 15) / 16;
  const int k0 = half * KH, k1 = min(ksteps, k0 + KH);           // this warp's steps of N
  // 16-token blocks that this warp finishes, and the blocks of M that it forms: row block, first column block, how many
  const int own0 = half ? 1 : 0, own1 = half ? 2 : 3;
  const int m_row = 0x03322110 >> 4 * warp & 15, m_col = 0x02002100 >> 4 * warp & 15, m_n = 0x02221111 >> 4 * warp & 15;
  bf* sm = reinterpret_cast<bf*>(smem);
  bf* sZ = sm + Cfg::OFF_Z;
  float* s_cs = reinterpret_cast<float*>(smem + Cfg::OFF_V * 2) + warp * 4 * SS_Q;
  float* s_dt = s_cs + SS_Q;
  float* s_e = s_dt + SS_Q;            // exp(cs)
  float* s_w = s_e + SS_Q;             // exp(cs_last - cs) dt
  float4* s_ex = reinterpret_cast<float4*>(smem + Cfg::OFF_X) + pw * 128 + lane;     // + receiving half * 512 + tile * 32
  const uint32_t a_sm = smem_u32(smem), a_z = smem_u32(sZ), a_m = a_sm + Cfg::OFF_M * 2, sc_ = a_sm + Cfg::OFF_C * 2;
  const bf* X = reinterpret_cast<const bf*>(p.x) + (long long)row0 * p.H * p.xp + h * p.xp;
  const bf* B = reinterpret_cast<const bf*>(p.b) + ((long long)row0 * p.G + grp) * p.np;
  const bf* Cc = reinterpret_cast<const bf*>(p.c) + ((long long)row0 * p.G + grp) * p.np;
  const bf* Z = reinterpret_cast<const bf*>(p.u) + (long long)row0 * p.u_ld + (long long)h * p.P;
  bf* Y = reinterpret_cast<bf*>(p.y) + (long long)row0 * p.y_ld + (long long)h * p.P;
  const bool z_vec = p.P % 8 == 0 && p.u_ld % 8 == 0 && (reinterpret_cast<uintptr_t>(p.u) & 15) == 0;
  const bool y_vec = p.P % 8 == 0 && p.y_ld % 8 == 0 && (reinterpret_cast<uintptr_t>(p.y) & 15) == 0;

  // rows of B or C: a thread keeps its piece of a row and steps through the rows
  auto load_n = [&](const bf* src, uint32_t dst, int t0) {
    constexpr int PR = KN * 2, RS = 256 / PR;            // 16-byte pieces of a row, rows per pass
    const int r0 = tid / PR, c = tid % PR * 8;
    const bf* s = src + (long long)(t0 + r0) * p.G * p.np + c;
    uint32_t d = dst + (r0 * Cfg::LN + c) * 2;
    const long long step = (long long)RS * p.G * p.np;
#pragma unroll
    for (int i = 0; i < SS_Q / RS; ++i, s += step, d += RS * Cfg::LN * 2) {
      const bool ok = t0 + r0 + i * RS < len && c < p.np;
      ss_cp16(d, ok ? s : src, ok);
    }
  };
  auto load_xb = [&](int ci) {
    if (ci < n_ch) {
      const int t0 = ci * SS_Q;
      const uint32_t st = a_sm + (ci & 1) * Cfg::STAGE * 2;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = i * 32 + half * 16 + (lane >> 1), c = c0 + (lane & 1) * 8;
        const bool ok = t0 + r < len && c < p.xp;
        ss_cp16(st + (r * SS_LX + pw * 16 + (lane & 1) * 8) * 2, ok ? X + (long long)(t0 + r) * p.H * p.xp + c : X, ok);
      }
      load_n(B, st + SS_Q * SS_LX * 2, t0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_c = [&](int ci) {
    if (ci < n_ch) load_n(Cc, sc_, ci * SS_Q);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // z of the rows and columns that this warp finishes
  auto load_z = [&](int t0) {
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int rb = (b ? own1 : own0) * 16;
      if (z_vec) {
        const int r = rb + (lane >> 1), c = c0 + (lane & 1) * 8;
        const bool ok = t0 + r < len && c < p.P;
        ss_cp16(a_z + (r * SS_LX + pw * 16 + (lane & 1) * 8) * 2, ok ? Z + (long long)(t0 + r) * p.u_ld + c : Z, ok);
      } else {
        for (int i = lane; i < 256; i += 32) {
          const int r = rb + (i >> 4), c = c0 + (i & 15);
          sZ[r * SS_LX + pw * 16 + (i & 15)] = t0 + r < len && c < p.P ? Z[(long long)(t0 + r) * p.u_ld + c] : __float2bfloat16_rn(0.f);
        }
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
  load_xb(0);
  if constexpr (!STATE) load_c(0);
  load_steps(0);
  // transposed state: column c0 + g + 8 (e >> 1), state row 16 k0 + 8 j + 2 t4 + (e & 1)
  float S[2 * KH][4];
  float* st = p.state + ((long long)P.rv.slot[seq] * p.H + h) * p.N * p.P;
  float* seg_st = p.n_seg ? p.seg_state + ((long long)z_id * p.H + h) * p.N * p.P : nullptr;
  const float* from = STATE ? nullptr : p.n_seg ? seg_st : P.rv.pos0[seq] == 0 ? nullptr : st;      // null: an empty state
#pragma unroll
  for (int j = 0; j < 2 * KH; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 16 * k0 + 8 * j + 2 * t4 + (e & 1), c = c0 + g + (e >> 1) * 8;
      S[j][e] = from && n < p.N && c < p.P ? from[(long long)n * p.P + c] : 0.f;
    }
  float la_sum = 0.f;
  const float D = p.D[h];
  // lane parts of the ldmatrix addresses: rows of a 16 x 16 tile whose quarters go (row 0, col 0), (0, 8), (8, 0), (8, 8) or
  // (0, 0), (8, 0), (0, 8), (8, 8)
  const int rc_r = (lane & 7) + (lane >> 4) * 8, rc_c = ((lane >> 3) & 1) * 8;
  const int cr_r = lane & 15, cr_c = (lane >> 4) * 8;

  for (int ci = 0; ci < n_ch; ++ci) {
    const int t0 = ci * SS_Q;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();             // the chunk is there, and everybody has left the previous one
    const uint32_t sx_ = a_sm + (ci & 1) * Cfg::STAGE * 2, sb_ = sx_ + SS_Q * SS_LX * 2;
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
      *reinterpret_cast<float2*>(s_e + 2 * lane) = make_float2(__expf(a - nla[1]), __expf(a));
      *reinterpret_cast<float2*>(s_w + 2 * lane) = make_float2(__expf(total - a + nla[1]) * ndt[0], __expf(total - a) * ndt[1]);
      __syncwarp();
    }
    la_sum += total;
    if constexpr (!STATE) load_z(t0);
    load_xb(ci + 1);
    load_steps(t0 + SS_Q);
    float Q[4][4];                // own tiles: two of block own0, two of block own1
    uint32_t x[4][4];             // x^T fragments: columns g (+ 8), tokens 16 kk + 2 t4 (+ 1) and 8 further
    if constexpr (!STATE) {
    // M: one or two 16 x 16 blocks per warp
    if (m_n > 0) {
      float G[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < KN; ++kk) {
        if (kk >= ksteps) break;
        uint32_t a[4], b[4], b2[4];
        ss_ldsm4(a, sc_ + ((m_row * 16 + cr_r) * Cfg::LN + kk * 16 + cr_c) * 2);
        ss_ldsm4(b, sb_ + ((m_col * 16 + rc_r) * Cfg::LN + kk * 16 + rc_c) * 2);
        ss_mma(G[0], a, b[0], b[1]);
        ss_mma(G[1], a, b[2], b[3]);
        if (m_n > 1) {
          ss_ldsm4(b2, sb_ + ((m_col * 16 + 16 + rc_r) * Cfg::LN + kk * 16 + rc_c) * 2);
          ss_mma(G[2], a, b2[0], b2[1]);
          ss_mma(G[3], a, b2[2], b2[3]);
        }
      }
      const float ct[2] = {s_cs[m_row * 16 + g], s_cs[m_row * 16 + g + 8]};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (i >= 2 * m_n) break;
        const int s = m_col * 16 + i * 8 + t4 * 2;
        const float2 cs = *reinterpret_cast<const float2*>(s_cs + s), dt = *reinterpret_cast<const float2*>(s_dt + s);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = m_row * 16 + g + 8 * r;
          const float m0 = s <= t ? G[i][2 * r] * __expf(ct[r] - cs.x) * dt.x : 0.f;
          const float m1 = s + 1 <= t ? G[i][2 * r + 1] * __expf(ct[r] - cs.y) * dt.y : 0.f;
          asm volatile("st.shared.b32 [%0], %1;" ::"r"(a_m + (t * SS_LX + s) * 2), "r"(pack_bf16x2(m0, m1)) : "memory");
        }
      }
    }
    // what this half of the state in front of the chunk contributes: S^T C^T
    float O[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) O[i][0] = O[i][1] = O[i][2] = O[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < KH; ++kk) {
      if (k0 + kk >= k1) break;
      uint32_t ah[4], al[4];
      split2(S[2 * kk][0], S[2 * kk][1], ah[0], al[0]);
      split2(S[2 * kk][2], S[2 * kk][3], ah[1], al[1]);
      split2(S[2 * kk + 1][0], S[2 * kk + 1][1], ah[2], al[2]);
      split2(S[2 * kk + 1][2], S[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        uint32_t b[4], b2[4];
        ss_ldsm4(b, sc_ + ((i * 16 + rc_r) * Cfg::LN + (k0 + kk) * 16 + rc_c) * 2);
        ss_ldsm4(b2, sc_ + ((i * 16 + 16 + rc_r) * Cfg::LN + (k0 + kk) * 16 + rc_c) * 2);
        ss_mma(O[2 * i], al, b[0], b[1]);
        ss_mma(O[2 * i + 1], al, b[2], b[3]);
        ss_mma(O[2 * i + 2], al, b2[0], b2[1]);
        ss_mma(O[2 * i + 3], al, b2[2], b2[3]);
        ss_mma(O[2 * i], ah, b[0], b[1]);
        ss_mma(O[2 * i + 1], ah, b[2], b[3]);
        ss_mma(O[2 * i + 2], ah, b2[0], b2[1]);
        ss_mma(O[2 * i + 3], ah, b2[2], b2[3]);
      }
    }
    // hand over the blocks that the other half finishes
    if (half) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int o = i < 2 ? i : i + 4;
        s_ex[i * 32] = make_float4(O[o][0], O[o][1], O[o][2], O[o][3]);
#pragma unroll
        for (int e = 0; e < 4; ++e) Q[i][e] = O[i + 2][e];
      }
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int o = i < 2 ? i : i + 4;
        s_ex[512 + i * 32] = make_float4(O[i + 2][0], O[i + 2][1], O[i + 2][2], O[i + 2][3]);
#pragma unroll
        for (int e = 0; e < 4; ++e) Q[i][e] = O[o][e];
      }
    }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) ss_ldsm4t(x[kk], sx_ + ((kk * 16 + rc_r) * SS_LX + pw * 16 + rc_c) * 2);
    if constexpr (!STATE) {
    __syncthreads();             // M and the exchange are complete, C and x are read
    load_c(ci + 1);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float4 v = s_ex[half * 512 + i * 32];
      const float2 e = *reinterpret_cast<const float2*>(s_e + (i < 2 ? own0 : own1) * 16 + (i & 1) * 8 + t4 * 2);
      Q[i][0] = (Q[i][0] + v.x) * e.x;
      Q[i][1] = (Q[i][1] + v.y) * e.y;
      Q[i][2] = (Q[i][2] + v.z) * e.x;
      Q[i][3] = (Q[i][3] + v.w) * e.y;
    }
    // what the chunk's own tokens contribute: x^T M^T
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk <= own0) {
        uint32_t b[4];
        ss_ldsm4(b, a_m + ((own0 * 16 + rc_r) * SS_LX + kk * 16 + rc_c) * 2);
        ss_mma(Q[0], x[kk], b[0], b[1]);
        ss_mma(Q[1], x[kk], b[2], b[3]);
      }
      if (kk <= own1) {
        uint32_t b[4];
        ss_ldsm4(b, a_m + ((own1 * 16 + rc_r) * SS_LX + kk * 16 + rc_c) * 2);
        ss_mma(Q[2], x[kk], b[0], b[1]);
        ss_mma(Q[3], x[kk], b[2], b[3]);
      }
    }
    }
    // this half of the state behind the chunk
    {
      const float f = __expf(total);
#pragma unroll
      for (int j = 0; j < 2 * KH; ++j) {
        S[j][0] *= f; S[j][1] *= f; S[j][2] *= f; S[j][3] *= f;
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t ah[4], al[4];
#pragma unroll
      for (int e = 0; e < 2; ++e) {          // tokens 16 kk + 8 e + 2 t4 and the next
        const int s = kk * 16 + 8 * e + t4 * 2;
        const float2 w = *reinterpret_cast<const float2*>(s_w + s);
        split2(lo_f(x[kk][2 * e]) * w.x, hi_f(x[kk][2 * e]) * w.y, ah[2 * e], al[2 * e]);
        split2(lo_f(x[kk][2 * e + 1]) * w.x, hi_f(x[kk][2 * e + 1]) * w.y, ah[2 * e + 1], al[2 * e + 1]);
      }
#pragma unroll
      for (int j = 0; j < KH; j += 2) {
        if (k0 + j >= k1) break;
        const bool two = j + 1 < KH && k0 + j + 1 < k1;
        uint32_t b[4], b2[4];
        ss_ldsm4t(b, sb_ + ((kk * 16 + cr_r) * Cfg::LN + (k0 + j) * 16 + cr_c) * 2);
        if (two) ss_ldsm4t(b2, sb_ + ((kk * 16 + cr_r) * Cfg::LN + (k0 + j + 1) * 16 + cr_c) * 2);
        ss_mma(S[2 * j], al, b[0], b[1]);
        ss_mma(S[2 * j + 1], al, b[2], b[3]);
        if (two) {
          ss_mma(S[(2 * j + 2) % (2 * KH)], al, b2[0], b2[1]);
          ss_mma(S[(2 * j + 3) % (2 * KH)], al, b2[2], b2[3]);
        }
        ss_mma(S[2 * j], ah, b[0], b[1]);
        ss_mma(S[2 * j + 1], ah, b[2], b[3]);
        if (two) {
          ss_mma(S[(2 * j + 2) % (2 * KH)], ah, b2[0], b2[1]);
          ss_mma(S[(2 * j + 3) % (2 * KH)], ah, b2[2], b2[3]);
        }
      }
    }
    if constexpr (STATE) continue;
    // skip connection and output gate in the fragment layout, then through the x columns of this warp's blocks to rows
    asm volatile("cp.async.wait_group 2;" ::: "memory");      // z; the next chunk may still be on its way
    __syncwarp();
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int kk = b ? own1 : own0;
      uint32_t z[4], xo[4], y[4];
      const uint32_t at = ((kk * 16 + rc_r) * SS_LX + pw * 16 + rc_c) * 2;
      ss_ldsm4t(z, a_z + at);
#pragma unroll
      for (int i = 0; i < 4; ++i) xo[i] = half ? x[1 + b][i] : x[3 * b][i];
#pragma unroll
      for (int i = 0; i < 4; ++i) {          // i = 2 (token half) + (column half)
        const float o0 = fmaf(D, lo_f(xo[i]), Q[2 * b + (i >> 1)][2 * (i & 1)]);
        const float o1 = fmaf(D, hi_f(xo[i]), Q[2 * b + (i >> 1)][2 * (i & 1) + 1]);
        y[i] = pack_bf16x2(o0 * silu_act<bf>(lo_f(z[i])), o1 * silu_act<bf>(hi_f(z[i])));
      }
      ss_stsm4t(sx_ + at, y[0], y[1], y[2], y[3]);
    }
    __syncwarp();
    const bf* sx_p = sm + (ci & 1) * Cfg::STAGE + pw * 16;
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int rb = (b ? own1 : own0) * 16;
      if (y_vec) {
        const int r = rb + (lane >> 1), c = (lane & 1) * 8;
        if (t0 + r < len && c0 + c < p.P)
          *reinterpret_cast<uint4*>(Y + (long long)(t0 + r) * p.y_ld + c0 + c) = *reinterpret_cast<const uint4*>(sx_p + r * SS_LX + c);
      } else {
        for (int i = lane; i < 256; i += 32) {
          const int r = rb + (i >> 4), c = i & 15;
          if (t0 + r < len && c0 + c < p.P) Y[(long long)(t0 + r) * p.y_ld + c0 + c] = sx_p[r * SS_LX + c];
        }
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 2 * KH; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 16 * k0 + 8 * j + 2 * t4 + (e & 1), c = c0 + g + (e >> 1) * 8;
      if (n < p.N && c < p.P && (STATE || last)) (STATE ? seg_st : st)[(long long)n * p.P + c] = S[j][e];
    }
  if (STATE && blockIdx.x == 0 && tid == 0) p.seg_la[(long long)z_id * p.H + h] = la_sum;
}

// What the segments of a sequence leave (from an empty state) -> the state in front of each.
__global__ void __launch_bounds__(256) ssd_chain_kernel(const SsdScanParams P) {
  const SxSsdArgs& p = P.a;
  const int h = blockIdx.y, seq = blockIdx.z, n = p.N * p.P, i = blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  float s = P.rv.pos0[seq] == 0 ? 0.f : p.state[((long long)P.rv.slot[seq] * p.H + h) * n + i];
  const int g0 = p.seg_first[seq], g1 = p.seg_first[seq + 1];
#pragma unroll 4
  for (int g = g0; g < g1; ++g) {
    float* at = p.seg_state + ((long long)g * p.H + h) * n + i;
    const float left = g + 1 < g1 ? *at : 0.f, f = g + 1 < g1 ? __expf(p.seg_la[(long long)g * p.H + h]) : 0.f;
    *at = s;
    s = fmaf(f, s, left);
  }
}

template <int KN, bool STATE>
static int launch_ssd_scan(const SsdScanParams& p, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(ssd_scan_kernel<KN, STATE>, cudaFuncAttributeMaxDynamicSharedMemorySize, SsdScanCfg<KN>::SMEM) != cudaSuccess) return -10;
    set = true;
  }
  ssd_scan_kernel<KN, STATE><<<dim3((p.a.P + 63) / 64, p.a.H, p.a.n_seg ? p.a.n_seg : p.rv.n), 256, SsdScanCfg<KN>::SMEM, st>>>(p);
  return last_rc();
}
template <int KN>
static int run_ssd_scan(const SsdScanParams& p, cudaStream_t st) {
  if (p.a.n_seg) {
    if (const int rc = launch_ssd_scan<KN, true>(p, st)) return rc;
    ssd_chain_kernel<<<dim3((p.a.N * p.a.P + 255) / 256, p.a.H, p.rv.n), 256, 0, st>>>(p);
  }
  return launch_ssd_scan<KN, false>(p, st);
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
  if (a->n_seg && (a->n_seg < a->ragged.n || a->n_seg > 65535 || a->seg_rows <= 0 || a->seg_rows % SS_Q || !a->seg_seq || !a->seg_first || !a->seg_state || !a->seg_la))
    return -1;
  if ((reinterpret_cast<uintptr_t>(a->x) | reinterpret_cast<uintptr_t>(a->b) | reinterpret_cast<uintptr_t>(a->c)) & 15) return -3;
  const SsdScanParams p{*a, view(&a->ragged)};
  if (a->N <= 32) return run_ssd_scan<2>(p, st);
  if (a->N <= 64) return run_ssd_scan<4>(p, st);
  if (a->N <= 128) return run_ssd_scan<8>(p, st);
  return run_ssd_scan<16>(p, st);
}
