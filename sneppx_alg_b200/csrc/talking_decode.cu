// Decode attention with a head mix in front of the softmax over the block pool (bf16): one query per sequence, keys limited
// to the query's chunk of positions.
//
// The mix is folded into the queries (sx_qkv_prep writes q'), so the scores of all heads are one product of q' [H, G d] with
// the cache rows as they lie in memory [keys, G d]. One CTA serves a slice of the visible keys of one sequence for all heads:
// cache rows stream through shared memory with cp.async, scores and P V run on tensor cores (mma.sync: the work is bound by
// reading the cache, the products are a few percent of it), and a second kernel merges the slices (talking_attn.cu).
#include "common.cuh"
#include "ragged.cuh"
#include "tc_common.cuh"
#include "sx_api.h"

namespace sx {

struct TalkDecParams {
  const __nv_bfloat16* qmix;  // [n, H, q_ld]
  const __nv_bfloat16* k; const __nv_bfloat16* v;   // cache rows [entries, G d], [entries, G dv]
  const int* block_table; const int* block_base;
  const __nv_bfloat16* gate;
  __nv_bfloat16* y;
  float* part;
  RaggedView rv;
  long long gate_ld, y_ld;
  int q_ld, table_ld, block_size, H, G, d, dv, size, splits, stages, ksplit;
  float scale, mul;
};

// shared-memory operands are 32-bit addresses: the inner loops then need no 64-bit address arithmetic
__device__ __forceinline__ void dec_cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(p) : "memory");
}
__device__ __forceinline__ void ldsm2(uint32_t (&r)[2], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(p) : "memory");
}
__device__ __forceinline__ void ldsm2t(uint32_t (&r)[2], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(p) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

constexpr int DW = 16, DT = DW * 32;     // warps and threads of a CTA

struct DecLayout {
  int HP, D16, ldq, ldk, ldv, ldp, lds, stage;   // elements (stage: bf16 elements of one K + V tile)
  int off_k, off_s, off_p, off_m, off_i, bytes;         // bytes
};
__host__ __device__ inline DecLayout dec_layout(int H, int G, int d, int dv, int KT, int stages, int ksplit) {
  DecLayout L;
  L.HP = (H + 15) / 16 * 16;
  L.D16 = (G * d + 15) / 16 * 16;
  L.ldq = L.D16 + 8;
  L.ldk = L.D16 + 8;
  L.ldv = G * dv + 8;
  L.ldp = KT + 8;
  L.lds = KT + 2;
  L.stage = KT * (L.ldk + L.ldv);
  L.off_k = L.HP * L.ldq * 2;
  L.off_s = L.off_k + stages * L.stage * 2;
  L.off_p = L.off_s + ksplit * L.HP * L.lds * 4;
  L.off_m = L.off_p + (L.HP + 16) * L.ldp * 2;
  L.off_i = L.off_m + 3 * L.HP * 4;
  L.bytes = L.off_i + G * (dv / 8) * 8;
  return L;
}

// QREG: every warp has one QK item of at most 8 k-steps, whose query fragments then stay in registers.
template <int KT, int MAXI, bool QREG>
__global__ void __launch_bounds__(DT) talk_decode_kernel(const TalkDecParams p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const DecLayout L = dec_layout(p.H, p.G, p.d, p.dv, KT, p.stages, p.ksplit);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* sKV = reinterpret_cast<__nv_bfloat16*>(smem + L.off_k);
  float* sS = reinterpret_cast<float*>(smem + L.off_s);
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(smem + L.off_p);
  float* sM = reinterpret_cast<float*>(smem + L.off_m);
  float* sL = sM + L.HP;
  float* sC = sL + L.HP;
  int2* sI = reinterpret_cast<int2*>(smem + L.off_i);   // P V items: first head of the group, value column
  const int n = blockIdx.x, split = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (p.rv.slot[n] < 0) return;            // padding row of a captured launch
  const int t = p.rv.cu[n], pos = p.rv.pos0[n];
  const int H = p.H, G = p.G, Gd = G * p.d, Gv = G * p.dv, grp = H / G;
  const int first = pos / p.size * p.size, n_vis = pos - first + 1;
  const int per = (n_vis + p.splits - 1) / p.splits;
  const int lo = first + split * per, hi = min(pos + 1, lo + per);
  const int n_tiles = hi > lo ? (hi - lo + KT - 1) / KT : 0;

  const int base = p.block_base[n];
  const int* table = p.block_table + (long long)n * p.table_ld;
  const int kc = Gd / 8, vc = Gv / 8;      // 16-byte pieces of a key / value row
  const uint32_t a_kv = smem_u32(sKV), stage_bytes = L.stage * 2, ldk_b = L.ldk * 2, ldv_b = L.ldv * 2;
  const uint32_t a_v = a_kv + KT * ldk_b;
  // rows past the end repeat the last key and are masked; lane i finds the entry of the warp's i-th row
  auto entry_of = [&](int tile) -> int {
    if (lane >= KT / DW || tile >= n_tiles) return 0;
    const int j = min(lo + tile * KT + warp + DW * lane, hi - 1), b = j / p.block_size;
    return table[b - base] * p.block_size + j - b * p.block_size;
  };
  auto fetch = [&](int tile, int stage, int e) {
    if (tile < n_tiles) {
      uint32_t dk = a_kv + stage * stage_bytes + warp * ldk_b + lane * 16, dv = a_v + stage * stage_bytes + warp * ldv_b + lane * 16;
#pragma unroll
      for (int i = 0; i < KT / DW; ++i) {
        const long long er = __shfl_sync(0xffffffffu, e, i);
        const __nv_bfloat16* kr = p.k + er * Gd + lane * 8;
        const __nv_bfloat16* vr = p.v + er * Gv + lane * 8;
        for (int c = 0; c < kc; c += 64) {
          if (c + lane < kc) dec_cp16(dk + c * 16, kr + c * 8);
          if (c + 32 + lane < kc) dec_cp16(dk + c * 16 + 512, kr + c * 8 + 256);
        }
        for (int c = 0; c < vc; c += 64) {
          if (c + lane < vc) dec_cp16(dv + c * 16, vr + c * 8);
          if (c + 32 + lane < vc) dec_cp16(dv + c * 16 + 512, vr + c * 8 + 256);
        }
        dk += DW * ldk_b;
        dv += DW * ldv_b;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  for (int s = 0; s < p.stages - 1; ++s) fetch(s, s, entry_of(s));
  int e_next = entry_of(p.stages - 1);       // one tile ahead of its use
  // queries, zero padding
  const __nv_bfloat16* q = p.qmix + (long long)t * H * p.q_ld;
  for (int i = tid; i < L.HP * (L.D16 / 8); i += DT) {
    const int h = i / (L.D16 / 8), c = i % (L.D16 / 8) * 8;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (h < H) x = *reinterpret_cast<const uint4*>(q + (long long)h * p.q_ld + c);
    *reinterpret_cast<uint4*>(sQ + h * L.ldq + c) = x;
  }
  if (Gd < L.D16)
    for (int i = tid; i < p.stages * KT * (L.D16 - Gd); i += DT) {
      const int w = L.D16 - Gd, s = i / (KT * w), r = i / w % KT;
      sKV[s * L.stage + r * L.ldk + Gd + i % w] = __float2bfloat16_rn(0.f);
    }
  for (int i = tid; i < (L.HP + 16) * L.ldp; i += DT) sP[i] = __float2bfloat16_rn(0.f);
  for (int i = tid; i < L.HP; i += DT) {
    sM[i] = -INFINITY;
    sL[i] = 0.f;
    sC[i] = 1.f;
  }
  const int nt8 = p.dv / 8, items = G * nt8, units = (KT / 8) * (L.HP / 16), ksteps = L.D16 / 16;
  for (int i = tid; i < items; i += DT) sI[i] = make_int2(i / nt8 * grp, i / nt8 * p.dv + i % nt8 * 8);
  float O[MAXI][4];
#pragma unroll
  for (int i = 0; i < MAXI; ++i) O[i][0] = O[i][1] = O[i][2] = O[i][3] = 0.f;

  // scores of a tile: (8 keys x 16 heads) units, each cut along k into ksplit parts
  uint32_t qf[QREG ? 8 : 1][4];
  if constexpr (QREG) {
    const int unit = warp % units, ks = warp / units, m0 = unit / (KT / 8) * 16, k0 = ksteps * ks / p.ksplit;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 8; ++kk) {
      qf[kk][0] = qf[kk][1] = qf[kk][2] = qf[kk][3] = 0;
      if (ks < p.ksplit && k0 + kk < ksteps * (ks + 1) / p.ksplit)
        ldsm4(qf[kk], smem_u32(sQ + (m0 + (lane & 15)) * L.ldq + (lane >> 4) * 8 + (k0 + kk) * 16));
    }
  }
  // item geometry of this warp's first (and with QREG only) item
  const int it_unit = warp % units, it_ks = warp / units;
  const int it_n0 = (it_unit % (KT / 8)) * 8, it_m0 = it_unit / (KT / 8) * 16;
  const int it_k0 = ksteps * it_ks / p.ksplit, it_k1 = ksteps * (it_ks + 1) / p.ksplit, it_nk = it_k1 - it_k0;
  const uint32_t a_kb = a_kv + ((it_n0 + (lane & 7)) * L.ldk + (lane >> 3) * 8 + it_k0 * 16) * 2;   // four 8-wide k pieces per load
  float* s_out = sS + (it_ks * L.HP + it_m0 + (lane >> 2)) * L.lds + it_n0 + (lane & 3) * 2;
  auto scores = [&](int stage) {
    if constexpr (QREG) {
      if (it_ks >= p.ksplit) return;
      float c[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
      const uint32_t kb = a_kb + stage * stage_bytes;
      if (it_nk == 8) {
        uint32_t b[4][4];                              // loads of all k-steps in flight together
#pragma unroll
        for (int i = 0; i < 4; ++i) ldsm4(b[i], kb + i * 64);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const uint32_t b0[2] = {b[i][0], b[i][1]}, b1[2] = {b[i][2], b[i][3]};
          mma16816(c[i & 1], qf[2 * i], b0);
          mma16816(c[2 + (i & 1)], qf[2 * i + 1], b1);
        }
      } else {
#pragma unroll
        for (int kk = 0; kk < 8; kk += 2) {
          if (kk + 1 < it_nk) {
            uint32_t b[4];
            ldsm4(b, kb + kk * 32);
            const uint32_t b0[2] = {b[0], b[1]}, b1[2] = {b[2], b[3]};
            mma16816(c[0], qf[kk], b0);
            mma16816(c[1], qf[kk + 1], b1);
          } else if (kk < it_nk) {
            uint32_t b[2];
            ldsm2(b, kb + kk * 32);
            mma16816(c[0], qf[kk], b);
          }
        }
      }
      *reinterpret_cast<float2*>(s_out) = make_float2((c[0][0] + c[1][0]) + (c[2][0] + c[3][0]), (c[0][1] + c[1][1]) + (c[2][1] + c[3][1]));
      *reinterpret_cast<float2*>(s_out + 8 * L.lds) =
          make_float2((c[0][2] + c[1][2]) + (c[2][2] + c[3][2]), (c[0][3] + c[1][3]) + (c[2][3] + c[3][3]));
    } else {
      for (int it = warp; it < units * p.ksplit; it += DW) {
        const int unit = it % units, ks = it / units, n0 = (unit % (KT / 8)) * 8, m0 = unit / (KT / 8) * 16;
        const int k0 = ksteps * ks / p.ksplit, k1 = ksteps * (ks + 1) / p.ksplit;
        const uint32_t qa = smem_u32(sQ + (m0 + (lane & 15)) * L.ldq + (lane >> 4) * 8);
        const uint32_t kb = a_kv + stage * stage_bytes + ((n0 + (lane & 7)) * L.ldk + (lane >> 3) * 8) * 2;
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
        int kk = k0;
#pragma unroll 4
        for (; kk + 1 < k1; kk += 2) {
          uint32_t a[4], a2[4], b[4];
          ldsm4(a, qa + kk * 32);
          ldsm4(a2, qa + kk * 32 + 32);
          ldsm4(b, kb + kk * 32);
          const uint32_t b0[2] = {b[0], b[1]}, b1[2] = {b[2], b[3]};
          mma16816(c0, a, b0);
          mma16816(c1, a2, b1);
        }
        if (kk < k1) {
          uint32_t a[4], b[2];
          ldsm4(a, qa + kk * 32);
          ldsm2(b, kb + kk * 32);
          mma16816(c0, a, b);
        }
        float* s = sS + (ks * L.HP + m0 + (lane >> 2)) * L.lds + n0 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(s) = make_float2(c0[0] + c1[0], c0[1] + c1[1]);
        *reinterpret_cast<float2*>(s + 8 * L.lds) = make_float2(c0[2] + c1[2], c0[3] + c1[3]);
      }
    }
  };
  auto arrived = [&]() {
    if (p.stages == 2) asm volatile("cp.async.wait_group 0;" ::: "memory");
    else asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
  };
  if (n_tiles > 0) {
    arrived();
    scores(0);
  }
  int stage = 0, refill = p.stages - 1;
  const uint32_t pv_a = smem_u32(sP + (lane & 15) * L.ldp + (lane >> 4) * 8), pv_b = a_v + (lane & 15) * ldv_b, ldp_b = L.ldp * 2;
  const int pr = lane >> 2;
  for (int tile = 0; tile < n_tiles; ++tile) {
    __syncthreads();          // scores of this tile are complete, and nobody reads the stage refilled next
    fetch(tile + p.stages - 1, refill, e_next);
    e_next = entry_of(tile + p.stages);
    const int next = stage + 1 == p.stages ? 0 : stage + 1;
    const int nk = min(KT, hi - lo - tile * KT);
    // two heads at a time, so that their reductions overlap
    for (int h0 = warp; h0 < H; h0 += 2 * DW) {
      const bool two = h0 + DW < H;
      float s[2], m_old[2], m[2], l[2];
      __nv_bfloat16 e[2];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int h = two ? h0 + DW * x : h0;
        s[x] = -INFINITY;
        if (lane < nk) {
          s[x] = 0.f;
          for (int ks = 0; ks < p.ksplit; ++ks) s[x] += sS[(ks * L.HP + h) * L.lds + lane];
          s[x] *= p.scale;
        }
        m_old[x] = sM[h];
        m[x] = s[x];
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int x = 0; x < 2; ++x) m[x] = fmaxf(m[x], __shfl_xor_sync(0xffffffffu, m[x], o));
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        m[x] = fmaxf(m_old[x], m[x]);
        e[x] = __float2bfloat16_rn(exp2f((s[x] - m[x]) * 1.4426950408889634f));
        l[x] = __bfloat162float(e[x]);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int x = 0; x < 2; ++x) l[x] += __shfl_xor_sync(0xffffffffu, l[x], o);
      __syncwarp();
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        if (x && !two) break;
        const int h = h0 + DW * x;
        if (lane < KT) sP[h * L.ldp + lane] = e[x];
        if (lane == 0) {
          const float c = exp2f((m_old[x] - m[x]) * 1.4426950408889634f);
          sC[h] = c;
          sM[h] = m[x];
          sL[h] = sL[h] * c + l[x];
        }
      }
    }
    if (tile + 1 < n_tiles) arrived();      // also: probabilities are visible
    else __syncthreads();
    const uint32_t sv = pv_b + stage * stage_bytes;
#pragma unroll
    for (int i0 = 0; i0 < MAXI; i0 += 4) {            // four items together: their loads overlap
      if (warp + i0 * DW >= items) break;
      uint32_t a[4][KT / 16][4], b[4][KT / 16][2];
      int2 w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) w[i] = sI[min(warp + (i0 + i) * DW, items - 1)];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) {
          ldsm4(a[i][kk], pv_a + w[i].x * ldp_b + kk * 32);
          ldsm2t(b[i][kk], sv + w[i].y * 2 + kk * 16 * ldv_b);
        }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (warp + (i0 + i) * DW >= items) break;
        const float f0 = pr < grp ? sC[w[i].x + pr] : 0.f;
        O[i0 + i][0] *= f0; O[i0 + i][1] *= f0;
        if (grp > 8) {
          const float f1 = pr + 8 < grp ? sC[w[i].x + pr + 8] : 0.f;
          O[i0 + i][2] *= f1; O[i0 + i][3] *= f1;
        }
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) mma16816(O[i0 + i], a[i][kk], b[i][kk]);
      }
    }
    if (tile + 1 < n_tiles) scores(next);
    refill = stage;
    stage = next;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < MAXI; ++i) {
    const int it = warp + i * DW;
    if (it >= items) break;
    const int j = it / nt8, c = (it % nt8) * 8 + (lane & 3) * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = (lane >> 2) + half * 8;
      if (r >= grp) continue;
      const int h = j * grp + r;
      const float a = O[i][2 * half], b = O[i][2 * half + 1];
      if (p.splits > 1) {
        float* o = p.part + (((long long)n * p.splits + split) * H + h) * (p.dv + 2) + 2 + c;
        o[0] = a;
        o[1] = b;
      } else {
        const float g = p.mul / ((1.f + __expf(-__bfloat162float(p.gate[(long long)t * p.gate_ld + h]))) * sL[h]);
        store2(p.y + (long long)t * p.y_ld + (long long)h * p.dv + c, a * g, b * g);
      }
    }
  }
  if (p.splits > 1)
    for (int h = tid; h < H; h += DT) {
      float* o = p.part + (((long long)n * p.splits + split) * H + h) * (p.dv + 2);
      o[0] = sM[h];
      o[1] = sL[h];
    }
}

struct DecPlan { int kt, stages, ksplit, maxi; };
static DecPlan dec_plan(int H, int G, int d, int dv) {
  DecPlan pl{0, 0, 0, 0};
  if (H <= 0 || G <= 0 || H % G || H / G > 16 || (G * d) % 8 || (d % 2) || dv % 8) return pl;
  const int per_warp = (G * (dv / 8) + DW - 1) / DW;
  if (per_warp > 16) return pl;
  for (int kt = 32; kt >= 16; kt -= 16)
    for (int stages = 3; stages >= 2; --stages) {
      const int units = (kt / 8) * ((H + 15) / 16), ks = units >= 16 ? 1 : (units >= 8 ? 2 : (units >= 4 ? 4 : 8));
      if (dec_layout(H, G, d, dv, kt, stages, ks).bytes <= 227 * 1024) return DecPlan{kt, stages, ks, per_warp <= 4 ? 4 : per_warp <= 8 ? 8 : 16};
    }
  return pl;
}

}  // namespace sx
using namespace sx;

// 1 when sx_talk_decode takes these sizes.
extern "C" int sx_talk_decode_ok(int H, int G, int d, int dv) { return dec_plan(H, G, d, dv).kt > 0; }

template <int KT, int MAXI, bool QREG>
static int launch_dec(const TalkDecParams& p, int n, int smem, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(talk_decode_kernel<KT, MAXI, QREG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -10;
    set = true;
  }
  talk_decode_kernel<KT, MAXI, QREG><<<dim3(n, p.splits), DT, smem, st>>>(p);
  return last_rc();
}

// Paged form only; `qmix` [n, H, q_ld] (zeros from G d up to the next multiple of 64). With splits > 1 the partial results go
// to a->part and the caller merges them (sx_talk_merge).
extern "C" int sx_talk_decode(const SxTalkArgs* a, const void* qmix, int q_ld, cudaStream_t st) {
  if (a->T <= 0) return 0;
  const DecPlan pl = dec_plan(a->H, a->G, a->d, a->dv);
  if (!pl.kt || !a->block_table || a->f32 || a->splits < 1) return -1;
  TalkDecParams p;
  p.qmix = (const __nv_bfloat16*)qmix; p.q_ld = q_ld; p.k = (const __nv_bfloat16*)a->k; p.v = (const __nv_bfloat16*)a->v;
  p.block_table = a->block_table; p.block_base = a->block_base; p.table_ld = a->table_ld; p.block_size = a->block_size;
  p.gate = (const __nv_bfloat16*)a->gate; p.gate_ld = a->gate_ld; p.y = (__nv_bfloat16*)a->y; p.y_ld = a->y_ld; p.part = a->part;
  p.rv = view(&a->ragged);
  p.H = a->H; p.G = a->G; p.d = a->d; p.dv = a->dv; p.size = a->size; p.splits = a->splits; p.stages = pl.stages; p.ksplit = pl.ksplit;
  p.scale = a->scale; p.mul = a->mul;
  const int smem = dec_layout(a->H, a->G, a->d, a->dv, pl.kt, pl.stages, pl.ksplit).bytes;
  int rc;
  const int units = (pl.kt / 8) * ((a->H + 15) / 16), ksteps = (a->G * a->d + 15) / 16;
  const bool qreg = pl.kt == 32 && pl.maxi == 4 && units * pl.ksplit <= DW && (ksteps + pl.ksplit - 1) / pl.ksplit <= 8;
  const int n = a->T;
  if (qreg) rc = launch_dec<32, 4, true>(p, n, smem, st);
  else if (pl.kt == 32) rc = pl.maxi == 4 ? launch_dec<32, 4, false>(p, n, smem, st) : pl.maxi == 8 ? launch_dec<32, 8, false>(p, n, smem, st) : launch_dec<32, 16, false>(p, n, smem, st);
  else rc = pl.maxi == 4 ? launch_dec<16, 4, false>(p, n, smem, st) : pl.maxi == 8 ? launch_dec<16, 8, false>(p, n, smem, st) : launch_dec<16, 16, false>(p, n, smem, st);
  if (rc == 0 && a->splits > 1) rc = sx_talk_merge(a, st);
  return rc;
}
