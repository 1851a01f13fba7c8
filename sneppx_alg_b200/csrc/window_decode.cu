// Decode form of window attention over tokens and averaged blocks (bf16): one query per sequence against the block pool; see
// window_attn.cu.
//
// A CTA serves a slice of the visible keys (averaged blocks, then window tokens) of one sequence for the query heads of one
// key head, up to 16 of them, padded to the 16 rows of an MMA. Its four warps take turns at tiles of 16 keys and do not wait
// for one another: each streams its tiles through its own ring in shared memory with cp.async and keeps its own maximum, sum
// and output accumulator in registers (mma.sync: the work is bound by reading the cache, the products are a few percent of
// it). The warps are merged at the end, the slices by sx_win_merge.
#include "tc_common.cuh"
#include "window_attn.cuh"

namespace sx {

constexpr int WD_T = 128, WD_STAGES = 3, WD_KEYS = 16;

template <int KD, int NV>      // k steps of 16 key entries, tiles of 8 value entries
struct WinDecCfg {
  static constexpr int LK = KD * 16 + 8, LV = NV * 8 + 8;       // row pitches (bf16 entries), free of bank conflicts
  static constexpr int STAGE = WD_KEYS * (LK + LV);
  static constexpr int SMEM = 4 * WD_STAGES * STAGE * 2;
  static constexpr int MERGE = 4 * 16 * (NV * 8 + 2) * 4;
  static_assert(MERGE <= SMEM && SMEM <= 227 * 1024, "shared memory");
};

__device__ __forceinline__ void wd_cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void wd_ldsm4(uint32_t (&r)[4], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(p) : "memory");
}
__device__ __forceinline__ void wd_ldsm4t(uint32_t (&r)[4], uint32_t p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(p) : "memory");
}
__device__ __forceinline__ void wd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

template <int KD, int NV>
__global__ void __launch_bounds__(WD_T) win_decode_kernel(const WinParams P, int head_parts) {
  using Cfg = WinDecCfg<KD, NV>;
  extern __shared__ __align__(128) uint8_t smem[];
  const SxWinAttnArgs& p = P.a;
  const int n = blockIdx.x, kvh = blockIdx.y / head_parts, part = blockIdx.y % head_parts, split = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  if (P.rv.slot[n] < 0) return;            // padding row of a captured launch
  const int row = P.rv.cu[n], pos = P.rv.pos0[n], grp = p.H / p.G, d = p.d, dv = p.dv;
  const int h0 = kvh * grp + part * 16, nh = min(16, grp - part * 16);
  const WinKeys keys = win_keys(pos, p.size, p.pool);
  const int total = keys.blocks + keys.tokens, per = (total + p.splits - 1) / p.splits;
  const int lo = min(total, split * per), hi = min(total, lo + per);
  const int n_tiles = (hi - lo + WD_KEYS - 1) / WD_KEYS;
  const int mine = n_tiles > warp ? (n_tiles - warp + 3) / 4 : 0;      // tiles of this warp: warp, warp + 4, ..

  __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(smem) + warp * WD_STAGES * Cfg::STAGE;
  const uint32_t a_ring = smem_u32(ring);
  const __nv_bfloat16* K = reinterpret_cast<const __nv_bfloat16*>(p.k) + kvh * d;
  const __nv_bfloat16* V = reinterpret_cast<const __nv_bfloat16*>(p.v) + kvh * dv;
  if (d % 16) {                            // the last k step reads 8 entries past the key: zeros
    for (int i = lane; i < WD_STAGES * WD_KEYS; i += 32)
      *reinterpret_cast<uint4*>(ring + i / WD_KEYS * Cfg::STAGE + i % WD_KEYS * Cfg::LK + d) = make_uint4(0, 0, 0, 0);
  }
  // lane i < 16 finds the entry of the tile's i-th key; keys past the end repeat the last one and are masked
  auto entry_of = [&](int k) -> long long {
    if (lane >= WD_KEYS || k >= mine) return 0;
    return win_entry(P, n, keys, min(lo + (warp + 4 * k) * WD_KEYS + lane, hi - 1));
  };
  auto fetch = [&](int k, long long e) {
    if (k < mine) {
      const uint32_t st = a_ring + (k % WD_STAGES) * Cfg::STAGE * 2;
      constexpr int KP = KD * 2;
#pragma unroll
      for (int i = 0; i < WD_KEYS * KP / 32; ++i) {
        const int r = (i * 32 + lane) / KP, c = (i * 32 + lane) % KP;
        const long long er = __shfl_sync(0xffffffffu, e, r);
        if (c * 8 < d) wd_cp16(st + (r * Cfg::LK + c * 8) * 2, K + er * p.k_ld + c * 8);
      }
#pragma unroll
      for (int i = 0; i < WD_KEYS * NV / 32; ++i) {
        const int r = (i * 32 + lane) / NV, c = (i * 32 + lane) % NV;
        const long long er = __shfl_sync(0xffffffffu, e, r);
        if (c * 8 < dv) wd_cp16(st + (WD_KEYS * Cfg::LK + r * Cfg::LV + c * 8) * 2, V + er * p.v_ld + c * 8);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int s = 0; s < WD_STAGES - 1; ++s) fetch(s, entry_of(s));
  long long e_next = entry_of(WD_STAGES - 1);       // one tile ahead of its use
  // query fragments, rows past the heads are zero
  uint32_t qf[KD][4];
  {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + ((long long)row * p.H + h0) * p.q_ld;
#pragma unroll
    for (int kk = 0; kk < KD; ++kk)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = g + (i & 1) * 8, c = kk * 16 + t4 * 2 + (i >> 1) * 8;
        qf[kk][i] = r < nh && c < p.q_ld ? *reinterpret_cast<const uint32_t*>(q + (long long)r * p.q_ld + c) : 0u;
      }
  }
  const int ksteps = (d + 15) / 16, vtiles = dv / 8;
  const float sl2 = p.scale * 1.4426950408889634f;
  float O[NV][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i) O[i][0] = O[i][1] = O[i][2] = O[i][3] = 0.f;
  const uint32_t k_lane = ((lane & 7) + (lane >> 4) * 8) * (Cfg::LK * 2) + ((lane >> 3) & 1) * 16;
  const uint32_t v_lane = WD_KEYS * Cfg::LK * 2 + (lane & 15) * (Cfg::LV * 2) + (lane >> 4) * 16;

  for (int k = 0; k < mine; ++k) {
    asm volatile("cp.async.wait_group %0;" ::"n"(WD_STAGES - 2) : "memory");
    __syncwarp();
    const uint32_t st = a_ring + (k % WD_STAGES) * Cfg::STAGE * 2;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int kk = 0; kk < KD; ++kk) {
      if (kk >= ksteps) break;
      uint32_t b[4];
      wd_ldsm4(b, st + k_lane + kk * 32);
      wd_mma(s[0], qf[kk], b[0], b[1]);
      wd_mma(s[1], qf[kk], b[2], b[3]);
    }
    fetch(k + WD_STAGES - 1, e_next);      // refills the stage of the tile before this one: all lanes are done with it
    e_next = entry_of(k + WD_STAGES);
    const int left = hi - lo - (warp + 4 * k) * WD_KEYS;       // keys of this tile that count
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[i][e] = i * 8 + t4 * 2 + (e & 1) < left ? s[i][e] * sl2 : -INFINITY;
        mx[e >> 1] = fmaxf(mx[e >> 1], s[i][e]);
      }
    bool grow = false;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      grow |= mx[r] > m[r] + 8.f;          // m = -inf at first; a tile always has a key
    }
    if (__any_sync(0xffffffffu, grow)) {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float nm = fmaxf(m[r], mx[r]), f = exp2f(m[r] - nm);
        m[r] = nm;
        l[r] *= f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          O[i][2 * r] *= f;
          O[i][2 * r + 1] *= f;
        }
      }
    }
    uint32_t pa[4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const uint32_t pb = pack_bf16x2(exp2f(s[i][2 * r] - m[r]), exp2f(s[i][2 * r + 1] - m[r]));
        pa[2 * i + r] = pb;
        l[r] += __uint_as_float(pb << 16) + __uint_as_float(pb & 0xffff0000u);
      }
#pragma unroll
    for (int i = 0; i < NV; i += 2) {
      if (i >= vtiles) break;
      uint32_t b[4];
      wd_ldsm4t(b, st + v_lane + i * 16);
      wd_mma(O[i], pa, b[0], b[1]);
      wd_mma(O[i + 1], pa, b[2], b[3]);
    }
    __syncwarp();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  __syncthreads();          // the rings are free
  float* buf = reinterpret_cast<float*>(smem);         // [4 warps][16 heads][max, sum, dv]
  const int ld = dv + 2;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float* b = buf + (warp * 16 + g + 8 * r) * ld;
    if (t4 == 0) {
      b[0] = m[r];
      b[1] = l[r];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (i < vtiles) {
        b[2 + i * 8 + t4 * 2] = O[i][2 * r];
        b[3 + i * 8 + t4 * 2] = O[i][2 * r + 1];
      }
  }
  __syncthreads();
  float* out = p.part + (((long long)n * p.splits + split) * p.H + h0) * ld;
  for (int i = tid; i < nh * ld; i += WD_T) {
    const int h = i / ld, c = i - h * ld;
    const float* b = buf + h * ld;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, b[w * 16 * ld]);
    float v = 0.f;
    if (c == 0) v = mm * 0.6931471805599453f;          // natural units for the merge
    else if (mm != -INFINITY)
#pragma unroll
      for (int w = 0; w < 4; ++w) v += b[w * 16 * ld + c] * exp2f(b[w * 16 * ld] - mm);
    out[i] = v;
  }
}

template <int KD, int NV>
static int launch_win_decode(const WinParams& p, cudaStream_t st) {
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(win_decode_kernel<KD, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, WinDecCfg<KD, NV>::SMEM) != cudaSuccess) return -10;
    set = true;
  }
  const int parts = (p.a.H / p.a.G + 15) / 16;
  win_decode_kernel<KD, NV><<<dim3(p.a.T, p.a.G * parts, p.a.splits), WD_T, WinDecCfg<KD, NV>::SMEM, st>>>(p, parts);
  return last_rc();
}
template <int KD>
static int pick_win_decode(const WinParams& p, cudaStream_t st) {
  return p.a.dv <= 64 ? launch_win_decode<KD, 8>(p, st) : p.a.dv <= 128 ? launch_win_decode<KD, 16>(p, st) : launch_win_decode<KD, 32>(p, st);
}

}  // namespace sx
using namespace sx;

// 1 when sx_win_decode takes these sizes.
extern "C" int sx_win_decode_ok(int H, int G, int d, int dv) {
  return H > 0 && G > 0 && H % G == 0 && d > 0 && d <= 256 && d % 8 == 0 && dv > 0 && dv <= 256 && dv % 8 == 0;
}

// Queries [T, H, q_ld] with zeros from d up to the next multiple of 16; partial results go to a->part and are merged into y.
extern "C" int sx_win_decode(const SxWinAttnArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (!sx_win_decode_ok(a->H, a->G, a->d, a->dv) || !a->block_table || !a->part || a->splits < 1 || a->q_ld % 2 || a->q_ld < (a->d + 15) / 16 * 16 ||
      !(a->scale > 0.f) || a->size <= 0 || a->pool <= 0)
    return -1;
  const WinParams p{*a, view(&a->ragged)};
  const int rc = a->d <= 64 ? pick_win_decode<4>(p, st) : a->d <= 128 ? pick_win_decode<8>(p, st) : pick_win_decode<16>(p, st);
  return rc ? rc : sx_win_merge(a, st);
}
