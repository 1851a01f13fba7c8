// Prompt form of window attention over tokens and averaged blocks on tcgen05 (bf16); see window_attn.cu.
//
// One CTA serves 128 query rows of one portion. It walks 128-key tiles, first those of the averaged blocks that its last row
// sees, then those of the tokens from its first row's window on, in two streams, each with its own scores, probabilities and
// output accumulator in TMEM and its own softmax warpgroup, so the tensor pipe works on one stream while the other does its
// softmax. PAIR: the streams are two heads of the same key head, which see the same keys, so every K and V tile is loaded once
// for both. Otherwise (an odd number of heads per key head) they are the even and the odd tiles of one head, merged at the end.
// The end also adds the sink, turns the outputs back by their row's angles and gates them.
//   S_x = Q_x K^T         over d in slices of 64: K by TMA in a ring of two-slice stages, Q resident in shared memory
//   P_x = exp2(S_x - m)   one query row per thread; packed bf16 over the S columns
//   O_x += P_x V          tcgen05.mma TS, V MN-major
// Keys are rows of a packed buffer: per sequence its averaged blocks, then its tokens in position order.
#include <limits.h>
#include "tc_common.cuh"
#include "tmap.h"
#include "window_attn.cuh"

namespace sx {

constexpr int WT_BM = 128, WT_BN = 128;
constexpr int WT_THREADS = 320;          // TMA warp, MMA warp, 2 x 4 softmax warps
constexpr int WT_SLICE = WT_BN * 128;    // bytes of a [128 x 64] bf16 slice
constexpr int WT_MAX_STAGES = 6;

struct WinTcParams {
  CUtensorMap tmQ, tmK, tmV;
  SxWinAttnArgs a;
  RaggedView rv;
  int nq, stages;
  float scale_log2;
};

// NQ: slices of a query row, 0 when only known at run time.
template <bool INTER, bool PAIR, int NQ>
__global__ void __launch_bounds__(WT_THREADS, 1) win_tc_kernel(const __grid_constant__ WinTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int stage_bytes = 2 * WT_SLICE;
  const int nq = NQ ? NQ : p.nq;
  uint8_t* sQ = smem;
  uint8_t* sR = smem + (PAIR ? 2 : 1) * nq * WT_SLICE;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sR + p.stages * stage_bytes);
  uint64_t* full = bars;                       // [stages]
  uint64_t* empty = bars + WT_MAX_STAGES;      // [stages]
  uint64_t* q_full = bars + 2 * WT_MAX_STAGES;
  uint64_t* s_full = q_full + 1;               // [2 streams]
  uint64_t* p_full = q_full + 3;
  uint64_t* o_done = q_full + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 7);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_ml = reinterpret_cast<float*>(sR);  // [2 streams][max, sum][128 rows], over the ring once it is drained

  const SxWinAttnArgs& a = p.a;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile = a.n_tiles - 1 - blockIdx.y, head0 = PAIR ? 2 * blockIdx.x : blockIdx.x;
  const int seq = a.tiles[2 * tile], r0 = a.tiles[2 * tile + 1];
  const int cu = p.rv.cu[seq], len = p.rv.cu[seq + 1] - cu, pos0 = p.rv.pos0[seq];
  const int t0 = cu + r0;
  const int p_first = pos0 + r0, p_last = pos0 + min(len, r0 + WT_BM) - 1;
  const WinKeys k_first = win_keys(p_first, a.size, a.pool), k_last = win_keys(p_last, a.size, a.pool);
  const int n_blk = (k_last.blocks + WT_BN - 1) / WT_BN;                        // tiles of averaged blocks
  const int n_steps = n_blk + (p_last - k_first.first) / WT_BN + 1;
  const int blk_row = a.pool_base[seq], tok_row = a.kv_base[seq] + k_first.first;
  const int kvh = head0 / (a.H / a.G);
  const int nv = (a.dv + 63) / 64;             // V slices

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

  // order of the ring. PAIR: K(0), then V(j), K(j + 1) for j = 0, 1, ..; else K(0), K(1), then V(j), K(j + 2)
  constexpr int AHEAD = PAIR ? 1 : 2;
  if (warp == 0) {
    if (lane == 0) {
      const int n_q = (PAIR ? 2 : 1) * nq;
      mbar_expect_tx(q_full, n_q * WT_SLICE);
      for (int c = 0; c < n_q; ++c) tma_load_2d(sQ + c * WT_SLICE, &p.tmQ, q_full, (head0 * nq + c) * 64, t0);
      int it = 0;
      bool ok = true;
      auto slot = [&](int bytes) -> int {      // waits for a free stage and announces `bytes`
        const int s = it % p.stages;
        ok = mbar_wait(&empty[s], ((it / p.stages) & 1) ^ 1, s_abort, a.status, ST_TIMEOUT_PRODUCER);
        if (ok) mbar_expect_tx(&full[s], bytes);
        ++it;
        return s;
      };
      auto row_of = [&](int j) { return j < n_blk ? blk_row + j * WT_BN : tok_row + (j - n_blk) * WT_BN; };
      auto load_k = [&](int j) {
        const int row = row_of(j);
        for (int c = 0; c < nq && ok; c += 2) {
          const int w = min(2, nq - c);
          const int s = slot(w * WT_SLICE);
          if (!ok) return;
          for (int e = 0; e < w; ++e) tma_load_2d(sR + s * stage_bytes + e * WT_SLICE, &p.tmK, &full[s], kvh * a.dp + (c + e) * 64, row);
        }
      };
      for (int j = 0; j < AHEAD && j < n_steps && ok; ++j) load_k(j);
      for (int j = 0; j < n_steps && ok; ++j) {
        const int s = slot(nv * WT_SLICE);
        if (!ok) break;
        const int row = row_of(j);
        for (int e = 0; e < nv; ++e) tma_load_2d(sR + s * stage_bytes + e * WT_SLICE, &p.tmV, &full[s], kvh * a.dvp + e * 64, row);
        if (j + AHEAD < n_steps) load_k(j + AHEAD);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_qk = umma_idesc_f16(WT_BM, WT_BN, 1, 0, 0);
      const uint32_t idesc_pv = umma_idesc_f16(WT_BM, (a.dv + 15) / 16 * 16, 1, 0, 1);
      int it = 0;
      bool ok = true;
      auto stage = [&]() -> int {
        const int s = it % p.stages;
        ok = mbar_wait(&full[s], (it / p.stages) & 1, s_abort, a.status, ST_TIMEOUT_MMA);
        ++it;
        return s;
      };
      // descriptors: an offset in bytes is added in units of 16 (addresses stay inside the 14-bit field)
      const uint64_t q_desc = umma_desc_sw128(smem_u32(sQ), 16, 1024), k_desc = umma_desc_sw128(smem_u32(sR), 16, 1024);
      const uint64_t v_desc = umma_desc_sw128(smem_u32(sR), WT_SLICE, 1024);
      // scores for stream x: query slices c, c + 1 with the K slices of stage s
      auto qk = [&](int x, int c, int s) {
        const uint32_t d = tmem_base + x * 256;
        const uint64_t qd = q_desc + (((PAIR ? x * nq : 0) + c) * WT_SLICE >> 4), kd = k_desc + (s * stage_bytes >> 4);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (c + e >= nq) break;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_f16_ss(d, qd + ((e * WT_SLICE + k * 32) >> 4), kd + ((e * WT_SLICE + k * 32) >> 4), idesc_qk, (c | e | k) ? 1u : 0u);
        }
      };
      auto pv = [&](int x, int s, bool first) {
        const uint32_t dO = tmem_base + x * 256 + 128, aP = tmem_base + x * 256;
        const uint64_t vd = v_desc + (s * stage_bytes >> 4);
#pragma unroll
        for (int k = 0; k < 8; ++k) umma_f16_ts(dO, aP + k * 8, vd + (k * 2048 >> 4), idesc_pv, (!first || k) ? 1u : 0u);
      };
      ok = mbar_wait(q_full, 0, s_abort, a.status, ST_TIMEOUT_MMA);
      if (ok) tc_fence_after();
      if constexpr (PAIR) {
        int k0 = 0, k1 = 0;                    // stages of the K tile in turn
        auto k_stages = [&]() {
          k0 = stage();
          if (nq > 2 && ok) k1 = stage();
          if (ok) tc_fence_after();
        };
        auto qk_all = [&](int x) {
          qk(x, 0, k0);
          if (nq > 2) qk(x, 2, k1);
          umma_commit(&s_full[x]);
        };
        auto k_release = [&]() {
          umma_commit(&empty[k0]);
          if (nq > 2) umma_commit(&empty[k1]);
        };
        if (ok) k_stages();
        if (ok) {
          qk_all(0);
          qk_all(1);
          k_release();
        }
        for (int j = 0; j < n_steps && ok; ++j) {
          const bool more = j + 1 < n_steps;
          const int s = stage();
          if (ok && more) k_stages();
          for (int x = 0; x < 2 && ok; ++x) {
            ok = mbar_wait(&p_full[x], j & 1, s_abort, a.status, ST_TIMEOUT_MMA);
            if (!ok) break;
            tc_fence_after();
            pv(x, s, j == 0);
            if (more) qk_all(x);
            else umma_commit(&o_done[x]);
          }
          if (!ok) break;
          umma_commit(&empty[s]);
          if (more) k_release();
        }
      } else {
        auto issue_qk = [&](int j) {
          for (int c = 0; c < nq; c += 2) {
            const int s = stage();
            if (!ok) return;
            tc_fence_after();
            qk(j & 1, c, s);
            umma_commit(&empty[s]);
          }
          umma_commit(&s_full[j & 1]);
        };
        if (ok) issue_qk(0);
        if (ok && n_steps > 1) issue_qk(1);
        for (int j = 0; j < n_steps && ok; ++j) {
          const int x = j & 1;
          const int s = stage();
          if (!ok) break;
          if (!mbar_wait(&p_full[x], (j >> 1) & 1, s_abort, a.status, ST_TIMEOUT_MMA)) break;
          tc_fence_after();
          pv(x, s, j < 2);
          umma_commit(&empty[s]);
          if (j + 2 >= n_steps) umma_commit(&o_done[x]);   // last step of this stream
          if (j + 2 < n_steps) issue_qk(j + 2);
        }
      }
    }
  } else {
    const int x = (warp - 2) >> 2;          // stream
    const int qd = warp & 3;                // TMEM lane quadrant of this warp
    const int row = qd * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(qd * 32) << 16;
    const uint32_t tS = tmem_base + x * 256 + lane_addr;
    const uint32_t tO = tS + 128;
    const bool row_ok = r0 + row < len;
    const WinKeys mine = win_keys(p_first + row, a.size, a.pool);
    float m_used = -INFINITY, l = 0.f;
    bool ok = true;
    const int head = head0 + (PAIR ? x : 0);
    int cnt = 0;                            // steps of this stream so far
    for (int j = PAIR ? 0 : x; j < n_steps; j += PAIR ? 1 : 2, ++cnt) {
      // key index of column 0, the indices that this row sees, and whether some row of the tile misses a column
      const bool is_blk = j < n_blk;
      const int kv0 = is_blk ? j * WT_BN : k_first.first + (j - n_blk) * WT_BN;
      const int lo = is_blk ? 0 : mine.first, hi = row_ok ? (is_blk ? mine.blocks : p_first + row + 1) : INT_MIN;
      const bool need_mask = r0 + WT_BM > len || (is_blk ? kv0 + WT_BN > k_first.blocks : kv0 + WT_BN - 1 > p_first || kv0 < k_last.first);
      if (!mbar_wait_warp(&s_full[x], cnt & 1, s_abort, a.status, ST_TIMEOUT_EPILOGUE)) { ok = false; break; }
      tc_fence_after();
      uint32_t r[WT_BN];
#pragma unroll
      for (int c = 0; c < WT_BN / 32; ++c) tmem_ld32(tS + c * 32, *reinterpret_cast<uint32_t(*)[32]>(&r[c * 32]));
      tmem_ld_wait();
      float mx = -INFINITY;
      if (need_mask) {
#pragma unroll
        for (int i = 0; i < WT_BN; ++i) {
          const int kv = kv0 + i;
          if (kv >= hi || kv < lo) r[i] = 0xff800000u;  // -inf
          mx = fmaxf(mx, __uint_as_float(r[i]));
        }
      } else {
#pragma unroll
        for (int i = 0; i < WT_BN; ++i) mx = fmaxf(mx, __uint_as_float(r[i]));
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
      for (int i = 0; i < WT_BN; i += 2) {
        const float v0 = exp2f(fmaf(__uint_as_float(r[i]), p.scale_log2, -m_sub));
        const float v1 = exp2f(fmaf(__uint_as_float(r[i + 1]), p.scale_log2, -m_sub));
        const uint32_t pb = pack_bf16x2(v0, v1);
        r[i / 2] = pb;
        lsum += __uint_as_float(pb << 16) + __uint_as_float(pb & 0xffff0000u);
      }
      l += lsum;
      // s_full(j) was committed after P V of this stream's previous step (in-order pipe): O and the S / P columns are ours
      if (cnt > 0 && __any_sync(0xffffffffu, rescale)) {
#pragma unroll 1
        for (int c = 0; c < (a.dv + 31) / 32; ++c) {
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
    const int n_streams = !PAIR && n_steps > 1 ? 2 : 1;      // accumulators that make up an output
    if constexpr (PAIR) {
      if (ok) ok = mbar_wait_warp(&o_done[x], 0, s_abort, a.status, ST_TIMEOUT_EPILOGUE);
    } else {
      for (int s = 0; s < n_streams && ok; ++s) ok = mbar_wait_warp(&o_done[s], 0, s_abort, a.status, ST_TIMEOUT_EPILOGUE);
      if (ok) {      // every load has been consumed: the ring is free
        s_ml[x * 2 * WT_BN + row] = m_used;
        s_ml[(x * 2 + 1) * WT_BN + row] = l;
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");      // the eight softmax warps
    }
    if (ok) {
      tc_fence_after();
      const float m0 = PAIR ? m_used : s_ml[row], l0 = PAIR ? l : s_ml[WT_BN + row];
      const float m1 = PAIR ? -INFINITY : s_ml[2 * WT_BN + row], l1 = PAIR ? 0.f : s_ml[3 * WT_BN + row];
      const float sk = a.sink[head] * 1.4426950408889634f;
      const float m = fmaxf(sk, fmaxf(m0, m1));
      const float e0 = m0 == -INFINITY ? 0.f : exp2f(m0 - m), e1 = m1 == -INFINITY ? 0.f : exp2f(m1 - m);
      const float inv = 1.f / (l0 * e0 + l1 * e1 + exp2f(sk - m));
      // a stream without a visible key for this row may hold anything finite; weight 0 removes it
      const float w0 = e0 * inv, w1 = e1 * inv;
      const long long t = t0 + row;
      const int half = a.dv / 2;
      const __nv_bfloat16* gr = reinterpret_cast<const __nv_bfloat16*>(a.gate) + t * a.gate_ld + (long long)head * a.dv;
      __nv_bfloat16* yr = reinterpret_cast<__nv_bfloat16*>(a.y) + t * a.y_ld + (long long)head * a.dv;
      const float2* turn = reinterpret_cast<const float2*>(a.turn) + t * half;
      const bool vec = half % 16 == 0 && a.y_ld % 8 == 0 && a.gate_ld % 8 == 0 &&
                       ((reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.gate) | reinterpret_cast<uintptr_t>(a.turn)) & 15) == 0;
      const uint32_t tO0 = PAIR ? tO : tmem_base + 128 + lane_addr, tO1 = tO0 + 256;
#pragma unroll 1
      for (int c = PAIR ? 0 : x; c < (half + 15) / 16; c += PAIR ? 1 : 2) {    // one stream: the warpgroups take turns
        const int ca = INTER ? c * 32 : c * 16, cb = INTER ? ca + 16 : half + c * 16;
        float v[32];
        {
          uint32_t o[16], o1[16];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            tmem_ld16(tO0 + (e ? cb : ca), o);
            if (n_streams > 1) tmem_ld16(tO1 + (e ? cb : ca), o1);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              v[e * 16 + i] = __uint_as_float(o[i]) * w0;
              if (n_streams > 1) v[e * 16 + i] = fmaf(__uint_as_float(o1[i]), w1, v[e * 16 + i]);
            }
          }
        }
        if (!row_ok) continue;
        // turn pair i back: (u, w) -> (u cos + w sin, w cos - u sin)
#pragma unroll
        for (int i = 0; i < 16; i += 2) {
          float4 cs = make_float4(0.f, 0.f, 0.f, 0.f);
          if (vec) {
            cs = *reinterpret_cast<const float4*>(turn + c * 16 + i);
          } else {
            if (c * 16 + i < half) { cs.x = turn[c * 16 + i].x; cs.y = turn[c * 16 + i].y; }
            if (c * 16 + i + 1 < half) { cs.z = turn[c * 16 + i + 1].x; cs.w = turn[c * 16 + i + 1].y; }
          }
          const int a0 = INTER ? 2 * i : i, b0 = INTER ? 2 * i + 1 : 16 + i, a1 = INTER ? 2 * i + 2 : i + 1, b1 = INTER ? 2 * i + 3 : 17 + i;
          const float u0 = v[a0], z0 = v[b0], u1 = v[a1], z1 = v[b1];
          v[a0] = u0 * cs.x + z0 * cs.y;
          v[b0] = z0 * cs.x - u0 * cs.y;
          v[a1] = u1 * cs.z + z1 * cs.w;
          v[b1] = z1 * cs.z - u1 * cs.w;
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int col = e ? cb : ca, end = INTER ? a.dv : (e ? a.dv : half);
          if (vec) {
#pragma unroll
            for (int i = 0; i < 16; i += 8) {
              const uint4 g = *reinterpret_cast<const uint4*>(gr + col + i);
              const uint32_t gw[4] = {g.x, g.y, g.z, g.w};
              uint32_t w[4];
#pragma unroll
              for (int k = 0; k < 4; ++k)
                w[k] = pack_bf16x2(__fdividef(v[e * 16 + i + 2 * k], 1.f + __expf(-__uint_as_float(gw[k] << 16))),
                                   __fdividef(v[e * 16 + i + 2 * k + 1], 1.f + __expf(-__uint_as_float(gw[k] & 0xffff0000u))));
              *reinterpret_cast<uint4*>(yr + col + i) = make_uint4(w[0], w[1], w[2], w[3]);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 16; ++i)
              if (col + i < end) yr[col + i] = __float2bfloat16_rn(v[e * 16 + i] / (1.f + __expf(-__bfloat162float(gr[col + i]))));
          }
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

static int win_rows_map(CUtensorMap* tm, const void* base, long long width, long long rows, long long ld) {
  uint64_t dims[2] = {(uint64_t)width, (uint64_t)rows};
  uint64_t strides[1] = {(uint64_t)ld * 2};
  uint32_t box[2] = {64, 128};
  return make_tmap(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, base, dims, strides, box);
}

template <bool INTER, bool PAIR, int NQ>
static int launch_win_tc(const WinTcParams& p, int smem, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(win_tc_kernel<INTER, PAIR, NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -10;
    set = true;
  }
  win_tc_kernel<INTER, PAIR, NQ><<<dim3(PAIR ? p.a.H / 2 : p.a.H, p.a.n_tiles), WT_THREADS, smem, st>>>(p);
  return last_rc();
}
template <bool INTER, bool PAIR>
static int pick_win_tc(const WinTcParams& p, int smem, cudaStream_t st) {
  return p.nq == 1 ? launch_win_tc<INTER, PAIR, 1>(p, smem, st) : p.nq == 2 ? launch_win_tc<INTER, PAIR, 2>(p, smem, st) : launch_win_tc<INTER, PAIR, 0>(p, smem, st);
}

}  // namespace sx
using namespace sx;

// 1 when sx_win_attn_tc takes these sizes.
extern "C" int sx_win_attn_tc_ok(int H, int G, int d, int dv) { return H > 0 && G > 0 && H % G == 0 && d > 0 && d <= 256 && dv > 0 && dv % 2 == 0 && dv <= 128; }

extern "C" int sx_win_attn_tc(const SxWinAttnArgs* a, cudaStream_t st) {
  if (a->n_tiles <= 0) return 0;
  if (!sx_win_attn_tc_ok(a->H, a->G, a->d, a->dv) || a->size <= 0 || a->pool <= 0 || !(a->scale > 0.f) || a->n_tiles > 65535) return -1;
  WinTcParams p;
  p.nq = (a->d + 63) / 64;
  if (a->k_ld % 8 || a->v_ld % 8 || a->dp % 8 || a->dvp % 8 || a->dp < a->d || a->dvp < a->dv || a->q_ld != p.nq * 64) return -3;
  int rc = win_rows_map(&p.tmQ, a->q, (long long)a->H * a->q_ld, a->T, (long long)a->H * a->q_ld);
  if (rc) return rc;
  rc = win_rows_map(&p.tmK, a->k, (long long)a->G * a->dp, a->kv_rows, a->k_ld);
  if (rc) return rc;
  rc = win_rows_map(&p.tmV, a->v, (long long)a->G * a->dvp, a->kv_rows, a->v_ld);
  if (rc) return rc;
  p.a = *a;
  p.rv = view(&a->ragged);
  p.scale_log2 = a->scale * 1.4426950408889634f;
  const bool pair = a->H / a->G % 2 == 0;
  const int held = (pair ? 2 : 1) * p.nq * WT_SLICE, room = 227 * 1024 - held - 1024 - 256;    // alignment and barriers set aside
  p.stages = room / (2 * WT_SLICE);
  if (p.stages > WT_MAX_STAGES) p.stages = WT_MAX_STAGES;
  if (p.stages < 1 + (p.nq + 1) / 2) return -4;          // a V tile and the next K tile are in the ring together
  const int smem = held + p.stages * 2 * WT_SLICE + 1024 + 256;
  if (pair) return a->interleaved ? pick_win_tc<true, true>(p, smem, st) : pick_win_tc<false, true>(p, smem, st);
  return a->interleaved ? pick_win_tc<true, false>(p, smem, st) : pick_win_tc<false, false>(p, smem, st);
}
