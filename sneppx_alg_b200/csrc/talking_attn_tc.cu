// Prompt attention with a head mix in front of the softmax, limited to chunks of positions, on tcgen05 (bf16).
//
// The mix score_h <- sum_g talk[h, g] (q_g . k_kv(g)) is linear, so it is folded into the queries: with
// q'_h = [ sum of talk[h, g] q_g over the query heads g of key head j ]_j, the mixed score of head h is q'_h . [k_0 .. k_G-1],
// one product over the concatenated key heads, and nothing couples the heads any more (sx_qkv_prep writes q').
//
// One CTA serves 128 query rows of one portion for one head and walks the visible 128-key tiles in two interleaved streams
// (even and odd tiles), each with its own scores, probabilities and output accumulator in TMEM and its own softmax
// warpgroup, so the tensor pipe works on one stream while the other does its softmax; the streams are merged at the end.
//   S_x = Q' K^T     over G d in slices of 64; K slices (and Q' slices when Q' does not stay resident) arrive by TMA in a
//                    ring of two-slice stages
//   P_x = exp2(S_x - m)   one query row per thread; packed bf16 over the S columns
//   O_x += P_x V     tcgen05.mma TS, V MN-major
// Keys are rows of a packed buffer in position order; a query at position p sees [floor(p / size) * size, p].
#include <limits.h>
#include "common.cuh"
#include "ragged.cuh"
#include "tc_common.cuh"
#include "tmap.h"
#include "sx_api.h"

namespace sx {

constexpr int TT_BM = 128, TT_BN = 128;
constexpr int TT_THREADS = 320;          // TMA warp, MMA warp, 2 x 4 softmax warps
constexpr int TT_SLICE = TT_BN * 128;    // bytes of a [128 x 64] bf16 slice
constexpr int TT_MAX_STAGES = 6;
constexpr int TT_RESIDENT = 8;           // slices of Q' that stay in shared memory

struct TalkTcParams {
  CUtensorMap tmQ, tmK, tmV;
  const int* tiles;           // [n_tiles, 2] portion, first row of it
  const int* kv_base;
  RaggedView rv;
  const __nv_bfloat16* gate;  // [T, gate_ld]
  __nv_bfloat16* y;
  int* status;
  long long gate_ld, y_ld;
  int H, grp, dv, dvp, nq, size, stages, resident, n_tiles;
  float scale_log2, mul;
};

__global__ void __launch_bounds__(TT_THREADS, 1) talk_tc_kernel(const __grid_constant__ TalkTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int stage_bytes = (p.resident ? 2 : 4) * TT_SLICE;   // K pair, and the matching Q' pair when it is streamed
  uint8_t* sQ = smem;
  uint8_t* sR = smem + (p.resident ? p.nq * TT_SLICE : 0);
  uint64_t* bars = reinterpret_cast<uint64_t*>(sR + p.stages * stage_bytes);
  uint64_t* full = bars;                       // [stages]
  uint64_t* empty = bars + TT_MAX_STAGES;      // [stages]
  uint64_t* q_full = bars + 2 * TT_MAX_STAGES;
  uint64_t* s_full = q_full + 1;               // [2 streams]
  uint64_t* p_full = q_full + 3;
  uint64_t* o_done = q_full + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 7);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_ml = reinterpret_cast<float*>(sR);  // [2 streams][max, sum][128 rows], over the ring once it is drained

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile = p.n_tiles - 1 - blockIdx.y, head = blockIdx.x;
  const int seq = p.tiles[2 * tile], r0 = p.tiles[2 * tile + 1];
  const int cu = p.rv.cu[seq], len = p.rv.cu[seq + 1] - cu, pos0 = p.rv.pos0[seq], base = p.kv_base[seq];
  const int t0 = cu + r0;
  const int p_first = pos0 + r0, p_last = pos0 + min(len, r0 + TT_BM) - 1;
  const int k_lo = p_first / p.size * p.size;
  const int n_steps = (p_last - k_lo) / TT_BN + 1;
  const int kvh = head / p.grp;
  const int nv = (p.dv + 63) / 64;             // V slices

  if (threadIdx.x == 0) {
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 4);
      mbar_init(&o_done[i], 1);
    }
    *s_abort = 0;
    mbar_fence_init();
    tma_prefetch_desc(&p.tmQ);
    tma_prefetch_desc(&p.tmK);
    tma_prefetch_desc(&p.tmV);
  }
  if (warp == 1) tmem_alloc(tmem_slot, 512);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  // order of the ring: K(0), K(1), then V(j), K(j + 2) for j = 0, 1, ..
  if (warp == 0) {
    if (lane == 0) {
      if (p.resident) {
        mbar_expect_tx(q_full, p.nq * TT_SLICE);
        for (int c = 0; c < p.nq; ++c) tma_load_2d(sQ + c * TT_SLICE, &p.tmQ, q_full, (head * p.nq + c) * 64, t0);
      }
      int it = 0;
      bool ok = true;
      auto slot = [&](int bytes) -> int {      // waits for a free stage and announces `bytes`
        const int s = it % p.stages;
        ok = mbar_wait(&empty[s], ((it / p.stages) & 1) ^ 1, s_abort, p.status, ST_TIMEOUT_PRODUCER);
        if (ok) mbar_expect_tx(&full[s], bytes);
        ++it;
        return s;
      };
      auto load_k = [&](int j) {
        const int row = base + k_lo + j * TT_BN;
        for (int c = 0; c < p.nq && ok; c += 2) {
          const int w = min(2, p.nq - c);
          const int s = slot(w * TT_SLICE * (p.resident ? 1 : 2));
          if (!ok) return;
          uint8_t* st = sR + s * stage_bytes;
          for (int e = 0; e < w; ++e) tma_load_2d(st + e * TT_SLICE, &p.tmK, &full[s], (c + e) * 64, row);
          if (!p.resident)
            for (int e = 0; e < w; ++e) tma_load_2d(st + (2 + e) * TT_SLICE, &p.tmQ, &full[s], (head * p.nq + c + e) * 64, t0);
        }
      };
      load_k(0);
      if (n_steps > 1 && ok) load_k(1);
      for (int j = 0; j < n_steps && ok; ++j) {
        const int s = slot(nv * TT_SLICE);
        if (!ok) break;
        for (int e = 0; e < nv; ++e)
          tma_load_2d(sR + s * stage_bytes + e * TT_SLICE, &p.tmV, &full[s], kvh * p.dvp + e * 64, base + k_lo + j * TT_BN);
        if (j + 2 < n_steps) load_k(j + 2);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_qk = umma_idesc_f16(TT_BM, TT_BN, 1, 0, 0);
      const uint32_t idesc_pv = umma_idesc_f16(TT_BM, (p.dv + 15) / 16 * 16, 1, 0, 1);
      int it = 0;
      bool ok = true;
      auto stage = [&]() -> int {
        const int s = it % p.stages;
        ok = mbar_wait(&full[s], (it / p.stages) & 1, s_abort, p.status, ST_TIMEOUT_MMA);
        ++it;
        return s;
      };
      auto issue_qk = [&](int j) {
        const uint32_t d = tmem_base + (j & 1) * 256;
        for (int c = 0; c < p.nq; c += 2) {
          const int s = stage();
          if (!ok) return;
          tc_fence_after();
          const uint32_t b0 = smem_u32(sR + s * stage_bytes);
          const uint32_t a0 = p.resident ? smem_u32(sQ + c * TT_SLICE) : b0 + 2 * TT_SLICE;
          for (int e = 0; e < 2 && c + e < p.nq; ++e)
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_f16_ss(d, umma_desc_sw128(a0 + e * TT_SLICE + k * 32, 16, 1024), umma_desc_sw128(b0 + e * TT_SLICE + k * 32, 16, 1024),
                          idesc_qk, (c | e | k) ? 1u : 0u);
          umma_commit(&empty[s]);
        }
        umma_commit(&s_full[j & 1]);
      };
      if (p.resident) ok = mbar_wait(q_full, 0, s_abort, p.status, ST_TIMEOUT_MMA);
      if (ok) {
        tc_fence_after();
        issue_qk(0);
      }
      if (ok && n_steps > 1) issue_qk(1);
      for (int j = 0; j < n_steps && ok; ++j) {
        const int x = j & 1;
        const int s = stage();
        if (!ok) break;
        if (!mbar_wait(&p_full[x], (j >> 1) & 1, s_abort, p.status, ST_TIMEOUT_MMA)) break;
        tc_fence_after();
        const uint32_t b0 = smem_u32(sR + s * stage_bytes);
        const uint32_t dO = tmem_base + x * 256 + 128, aP = tmem_base + x * 256;
#pragma unroll
        for (int k = 0; k < 8; ++k)
          umma_f16_ts(dO, aP + k * 8, umma_desc_sw128(b0 + k * 2048, TT_SLICE, 1024), idesc_pv, (j > 1 || k) ? 1u : 0u);
        umma_commit(&empty[s]);
        if (j + 2 >= n_steps) umma_commit(&o_done[x]);   // last step of this stream
        if (j + 2 < n_steps) issue_qk(j + 2);
      }
    }
  } else {
    const int x = (warp - 2) >> 2;          // stream
    const int qd = warp & 3;                // TMEM lane quadrant of this warp
    const int row = qd * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(qd * 32) << 16;
    const uint32_t tS = tmem_base + x * 256 + lane_addr;
    const uint32_t tO = tS + 128;
    const int pos = p_first + row;
    const bool row_ok = r0 + row < len;
    const int hi_k = row_ok ? pos : -1, lo_k = pos / p.size * p.size;
    const int tile_lo_max = p_last / p.size * p.size;     // latest chunk start of the tile's rows
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = x; j < n_steps; j += 2) {
      const int kv0 = k_lo + j * TT_BN;
      if (!mbar_wait_warp(&s_full[x], (j >> 1) & 1, s_abort, p.status, ST_TIMEOUT_EPILOGUE)) { ok = false; break; }
      tc_fence_after();
      const bool need_mask = kv0 + TT_BN - 1 > p_first || kv0 < tile_lo_max || r0 + TT_BM > len;
      uint32_t r[TT_BN];
#pragma unroll
      for (int c = 0; c < TT_BN / 32; ++c) tmem_ld32(tS + c * 32, *reinterpret_cast<uint32_t(*)[32]>(&r[c * 32]));
      tmem_ld_wait();
      float mx = -INFINITY;
      if (need_mask) {
#pragma unroll
        for (int i = 0; i < TT_BN; ++i) {
          const int kv = kv0 + i;
          if (kv > hi_k || kv < lo_k) r[i] = 0xff800000u;  // -inf
          mx = fmaxf(mx, __uint_as_float(r[i]));
        }
      } else {
#pragma unroll
        for (int i = 0; i < TT_BN; ++i) mx = fmaxf(mx, __uint_as_float(r[i]));
      }
      mx *= p.scale_log2;
      float alpha = 1.f;
      bool rescale = false;
      if ((mx > m_used + 8.f || m_used == -INFINITY) && mx != -INFINITY) {
        alpha = (m_used == -INFINITY) ? 0.f : exp2f(m_used - mx);
        rescale = (m_used != -INFINITY);
        m_used = mx;
      }
      l *= alpha;
      const float m_sub = (m_used == -INFINITY) ? 0.f : m_used;
      float lsum = 0.f;
#pragma unroll
      for (int i = 0; i < TT_BN; i += 2) {
        const float v0 = exp2f(fmaf(__uint_as_float(r[i]), p.scale_log2, -m_sub));
        const float v1 = exp2f(fmaf(__uint_as_float(r[i + 1]), p.scale_log2, -m_sub));
        const uint32_t pb = pack_bf16x2(v0, v1);
        r[i / 2] = pb;
        lsum += __uint_as_float(pb << 16) + __uint_as_float(pb & 0xffff0000u);
      }
      l += lsum;
      // s_full(j) was committed after P V of this stream's previous step (in-order pipe): O and the S / P columns are ours
      if (j > 1 && __any_sync(0xffffffffu, rescale)) {
#pragma unroll 1
        for (int c = 0; c < (p.dv + 31) / 32; ++c) {
          uint32_t o[32];
          tmem_ld32(tO + c * 32, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
          tmem_st32(tO + c * 32, o);
        }
      }
      tmem_st32(tS, *reinterpret_cast<uint32_t(*)[32]>(&r[0]));
      tmem_st32(tS + 32, *reinterpret_cast<uint32_t(*)[32]>(&r[32]));
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[x]);
    }
    const int n_streams = n_steps > 1 ? 2 : 1;
    for (int s = 0; s < n_streams && ok; ++s) ok = mbar_wait_warp(&o_done[s], 0, s_abort, p.status, ST_TIMEOUT_EPILOGUE);
    if (ok) {      // every load has been consumed: the ring is free
      s_ml[x * 2 * TT_BM + row] = m_used;
      s_ml[(x * 2 + 1) * TT_BM + row] = l;
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");      // the eight softmax warps
    if (ok) {
      tc_fence_after();
      const float m0 = s_ml[row], l0 = s_ml[TT_BM + row], m1 = s_ml[2 * TT_BM + row], l1 = s_ml[3 * TT_BM + row];
      const float m = fmaxf(m0, m1);
      const float e0 = m0 == -INFINITY ? 0.f : exp2f(m0 - m), e1 = m1 == -INFINITY ? 0.f : exp2f(m1 - m);
      const float den = l0 * e0 + l1 * e1;
      const long long t = t0 + row;
      float g = 0.f;
      if (row_ok) g = p.mul / (1.f + __expf(-__bfloat162float(p.gate[t * p.gate_ld + head])));
      const float inv = den > 0.f ? g / den : 0.f;
      const float w0 = e0 * inv, w1 = e1 * inv;
      __nv_bfloat16* yr = p.y + t * p.y_ld + (long long)head * p.dv;
      const bool vec = (p.dv % 8 == 0) && (p.y_ld % 8 == 0) && ((reinterpret_cast<uintptr_t>(p.y) & 15) == 0);
      const uint32_t tO0 = tmem_base + 128 + lane_addr, tO1 = tO0 + 256;
#pragma unroll 1
      for (int c = x; c < (p.dv + 15) / 16; c += 2) {    // each warpgroup writes every other 16 columns
        uint32_t a[16], b[16];
        tmem_ld16(tO0 + c * 16, a);
        if (n_streams > 1) tmem_ld16(tO1 + c * 16, b);
        tmem_ld_wait();
        float v[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          // a stream without a visible key for this row may hold anything finite; weight 0 removes it
          v[i] = __uint_as_float(a[i]) * w0;
          if (n_streams > 1) v[i] = fmaf(__uint_as_float(b[i]), w1, v[i]);
        }
        if (!row_ok) continue;
        if (vec) {
#pragma unroll
          for (int i = 0; i < 16; i += 8) {
            if (c * 16 + i >= p.dv) break;
            uint4 w;
            w.x = pack_bf16x2(v[i], v[i + 1]);
            w.y = pack_bf16x2(v[i + 2], v[i + 3]);
            w.z = pack_bf16x2(v[i + 4], v[i + 5]);
            w.w = pack_bf16x2(v[i + 6], v[i + 7]);
            *reinterpret_cast<uint4*>(yr + c * 16 + i) = w;
          }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (c * 16 + i < p.dv) yr[c * 16 + i] = __float2bfloat16_rn(v[i]);
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*s_abort) bounded_delay_ns(2000000);
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

static int make_rows_map(CUtensorMap* tm, const void* base, long long width, long long rows, long long ld) {
  uint64_t dims[2] = {(uint64_t)width, (uint64_t)rows};
  uint64_t strides[1] = {(uint64_t)ld * 2};
  uint32_t box[2] = {64, 128};
  return make_tmap(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, base, dims, strides, box);
}

}  // namespace sx
using namespace sx;

// 1 when sx_talk_attn_tc takes these sizes.
extern "C" int sx_talk_attn_tc_ok(int H, int G, int d, int dv) { return H > 0 && G > 0 && H % G == 0 && d % 2 == 0 && dv <= 128; }

extern "C" int sx_talk_attn_tc(const SxTalkTcArgs* a, cudaStream_t st) {
  if (a->n_tiles <= 0) return 0;
  if (!sx_talk_attn_tc_ok(a->H, a->G, a->d, a->dv)) return -1;
  if (a->k_ld % 8 || a->v_ld % 8 || a->dvp % 8) return -3;
  TalkTcParams p;
  p.nq = (a->G * a->d + 63) / 64;
  int rc = make_rows_map(&p.tmQ, a->qmix, (long long)a->H * p.nq * 64, a->T, (long long)a->H * p.nq * 64);
  if (rc) return rc;
  rc = make_rows_map(&p.tmK, a->k, (long long)a->G * a->d, a->kv_rows, a->k_ld);
  if (rc) return rc;
  rc = make_rows_map(&p.tmV, a->v, (long long)a->G * a->dvp, a->kv_rows, a->v_ld);
  if (rc) return rc;
  p.tiles = a->tiles; p.kv_base = a->kv_base; p.rv = view(&a->ragged);
  p.gate = (const __nv_bfloat16*)a->gate; p.gate_ld = a->gate_ld; p.y = (__nv_bfloat16*)a->y; p.y_ld = a->y_ld;
  p.status = a->status;
  p.H = a->H; p.grp = a->H / a->G; p.dv = a->dv; p.dvp = a->dvp; p.size = a->size; p.n_tiles = a->n_tiles;
  p.scale_log2 = a->scale * 1.4426950408889634f; p.mul = a->mul;
  p.resident = p.nq <= TT_RESIDENT;
  const int stage = (p.resident ? 2 : 4) * TT_SLICE, held = p.resident ? p.nq * TT_SLICE : 0;
  const int room = 227 * 1024 - held - 1024 - 256;    // alignment and barriers set aside
  p.stages = room / stage;
  if (p.stages > TT_MAX_STAGES) p.stages = TT_MAX_STAGES;
  const int smem = held + p.stages * stage + 1024 + 256;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(talk_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -10;
    set = true;
  }
  if (smem > 227 * 1024) return -4;
  talk_tc_kernel<<<dim3(a->H, a->n_tiles), TT_THREADS, smem, st>>>(p);
  return last_rc();
}
