// Attention with a head mix in front of the softmax, limited to chunks of positions, SIMT form: any head count and size,
// 32-bit or bf16 keys and values, packed rows (prompts) or the block pool (decoding).
//
// One CTA serves one query row for all heads: the mix couples the heads, so the raw scores of a key tile for every head
// sit side by side in shared memory, are mixed there, and go through an online softmax per head. The visible keys of a
// query at position p are [floor(p / size) * size, p]; with `splits` > 1 that range is cut into equal parts served by
// different CTAs whose partial results a second kernel merges.
#include "common.cuh"
#include "ragged.cuh"
#include "sx_api.h"

namespace sx {

constexpr int TA_KT = 32;     // keys per tile

struct TalkParams {
  SxTalkArgs a;
  RaggedView rv;
};

template <typename A>
__device__ __forceinline__ float dot_row(const float* __restrict__ q, const A* __restrict__ k, int d) {
  float acc = 0.f;
  for (int i = 0; i < d; i += 2) {
    acc = fmaf(q[i], to_f(k[i]), acc);
    acc = fmaf(q[i + 1], to_f(k[i + 1]), acc);
  }
  return acc;
}

template <typename A, bool PAGED>
__global__ void __launch_bounds__(256) talk_attn_kernel(const TalkParams P) {
  const SxTalkArgs& p = P.a;
  extern __shared__ __align__(16) float sm[];
  const int H = p.H, G = p.G, d = p.d, dv = p.dv, grp = H / G;
  float* sq = sm;                       // [H, d]
  float* st = sq + H * d;               // [H, H]
  float* raw = st + H * H;              // [H, KT]
  float* pr = raw + H * TA_KT;          // [H, KT]
  float* so = pr + H * TA_KT;           // [H, dv]
  float* sm_m = so + H * dv;            // [H]
  float* sm_l = sm_m + H;               // [H]
  float* sm_c = sm_l + H;               // [H]
  const int t = blockIdx.x, split = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = P.rv.tok_seq[t], pos = P.rv.tok_pos[t];
  if (P.rv.slot[seq] < 0) return;
  const int first = pos / p.size * p.size, n_vis = pos - first + 1;
  const int per = (n_vis + p.splits - 1) / p.splits;
  const int lo = first + split * per, hi = min(pos + 1, lo + per);
  for (int i = tid; i < H * d; i += 256) sq[i] = p.q[(long long)t * H * d + i] * p.scale;
  for (int i = tid; i < H * H; i += 256) st[i] = p.talk[i];
  for (int i = tid; i < H * dv; i += 256) so[i] = 0.f;
  for (int i = tid; i < H; i += 256) {
    sm_m[i] = -INFINITY;
    sm_l[i] = 0.f;
  }
  const A* K = reinterpret_cast<const A*>(p.k);
  const A* V = reinterpret_cast<const A*>(p.v);
  auto entry = [&](int j) -> long long {
    if constexpr (PAGED)
      return (long long)p.block_table[(long long)seq * p.table_ld + j / p.block_size - p.block_base[seq]] * p.block_size + j % p.block_size;
    else
      return (long long)p.kv_base[seq] + j;
  };
  for (int j0 = lo; j0 < hi; j0 += TA_KT) {
    const int nk = min(TA_KT, hi - j0);
    __syncthreads();
    for (int i = tid; i < H * TA_KT; i += 256) {
      const int h = i / TA_KT, j = i % TA_KT;
      if (j < nk) raw[i] = dot_row<A>(sq + h * d, K + entry(j0 + j) * p.k_ld + (h / grp) * d, d);
    }
    __syncthreads();
    for (int i = tid; i < H * TA_KT; i += 256) {
      const int h = i / TA_KT, j = i % TA_KT;
      float s = -INFINITY;
      if (j < nk) {
        s = 0.f;
        for (int g = 0; g < H; ++g) s = fmaf(st[h * H + g], raw[g * TA_KT + j], s);
      }
      pr[i] = s;
    }
    __syncthreads();
    for (int h = warp; h < H; h += 8) {
      const float s = pr[h * TA_KT + lane];
      const float m_old = sm_m[h], m = fmaxf(m_old, warp_max(s));
      const float e = expf(s - m);
      const float l = warp_sum(e);
      pr[h * TA_KT + lane] = e;
      if (lane == 0) {
        const float c = expf(m_old - m);
        sm_c[h] = c;
        sm_m[h] = m;
        sm_l[h] = sm_l[h] * c + l;
      }
    }
    __syncthreads();
    for (int i = tid; i < H * dv; i += 256) {
      const int h = i / dv, c = i % dv;
      float acc = so[i] * sm_c[h];
      const A* vc = V + (h / grp) * p.dvp + c;
      for (int j = 0; j < nk; ++j) acc = fmaf(pr[h * TA_KT + j], to_f(vc[entry(j0 + j) * p.v_ld]), acc);
      so[i] = acc;
    }
  }
  __syncthreads();
  if (p.splits > 1) {
    float* part = p.part + ((long long)t * p.splits + split) * H * (dv + 2);
    for (int i = tid; i < H * dv; i += 256) part[(i / dv) * (dv + 2) + 2 + i % dv] = so[i];
    for (int h = tid; h < H; h += 256) {
      part[h * (dv + 2)] = sm_m[h];
      part[h * (dv + 2) + 1] = sm_l[h];
    }
    return;
  }
  A* y = reinterpret_cast<A*>(p.y) + (long long)t * p.y_ld;
  const A* gate = reinterpret_cast<const A*>(p.gate) + (long long)t * p.gate_ld;
  for (int i = tid; i < H * dv; i += 256) {
    const int h = i / dv;
    y[i] = from_f<A>(so[i] / sm_l[h] * (sigmoid_f(to_f(gate[h])) * p.mul));
  }
}

template <typename A>
__global__ void __launch_bounds__(128) talk_merge_kernel(const TalkParams P) {
  const SxTalkArgs& p = P.a;
  const int h = blockIdx.x, t = blockIdx.y, dv = p.dv;
  if (P.rv.slot[P.rv.tok_seq[t]] < 0) return;
  const float* part = p.part + ((long long)t * p.splits * p.H + h) * (dv + 2);
  const long long sstep = (long long)p.H * (dv + 2);
  float m = -INFINITY;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, part[s * sstep]);
  float l = 0.f;
  for (int s = 0; s < p.splits; ++s) l += part[s * sstep + 1] * expf(part[s * sstep] - m);
  const float gate = sigmoid_f(to_f(reinterpret_cast<const A*>(p.gate)[(long long)t * p.gate_ld + h])) * p.mul / l;
  for (int c = threadIdx.x; c < dv; c += 128) {
    float acc = 0.f;
    for (int s = 0; s < p.splits; ++s) acc = fmaf(part[s * sstep + 2 + c], expf(part[s * sstep] - m), acc);
    reinterpret_cast<A*>(p.y)[(long long)t * p.y_ld + (long long)h * dv + c] = from_f<A>(acc * gate);
  }
}

}  // namespace sx
using namespace sx;

template <typename A>
static int launch_talk(const TalkParams& P, cudaStream_t st) {
  const SxTalkArgs& a = P.a;
  const int smem = (a.H * a.d + a.H * a.H + 2 * a.H * TA_KT + a.H * a.dv + 3 * a.H) * 4;
  if (smem > 227 * 1024) return -2;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(talk_attn_kernel<A, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(talk_attn_kernel<A, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess)
      return -10;
    set = true;
  }
  const dim3 grid(a.T, a.splits);
  if (a.block_table) talk_attn_kernel<A, true><<<grid, 256, smem, st>>>(P);
  else talk_attn_kernel<A, false><<<grid, 256, smem, st>>>(P);
  if (a.splits > 1) talk_merge_kernel<A><<<dim3(a.H, a.T), 128, 0, st>>>(P);
  return last_rc();
}

// Merges the partial results of a->splits key slices per query into y.
extern "C" int sx_talk_merge(const SxTalkArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  TalkParams P;
  P.a = *a;
  P.rv = view(&a->ragged);
  SX_ACT_DISPATCH(a->f32, (talk_merge_kernel<A><<<dim3(a->H, a->T), 128, 0, st>>>(P)));
  return last_rc();
}

extern "C" int sx_talk_attn(const SxTalkArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (a->G <= 0 || a->H % a->G || a->d % 2 || a->size <= 0 || a->splits < 1) return -1;
  TalkParams P;
  P.a = *a;
  P.rv = view(&a->ragged);
  SX_ACT_DISPATCH(a->f32, { return launch_talk<A>(P, st); });
  return 0;
}
