// Row-wise pieces of a decoder whose residual stream is kept in fp32 and whose batches are ragged (token rows of several
// sequences packed one after another): embedding, RMSNorm, per-head output norm with gate, short causal convolution
// with carried inputs, query / key preparation.
//
// Every kernel is templated on the activation type A (bf16 in serving, float for 32-bit runs). Arithmetic is fp32
// throughout; only what is stored as an activation is rounded to A.
#include "common.cuh"
#include "ragged.cuh"
#include "sx_api.h"

namespace sx {

// ------------------------------------------------------------------ embedding
template <typename A>
__global__ void embed_f32_kernel(const A* __restrict__ table, const int* __restrict__ ids, float* __restrict__ x, int width) {
  const A* src = table + (long long)ids[blockIdx.x] * width;
  float* dst = x + (long long)blockIdx.x * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = to_f(src[i]);
}

// ------------------------------------------------------------------ RMSNorm of fp32 rows
// rows: optional list of source rows (out row r = norm of x[rows[r]]).
template <typename A>
__global__ void __launch_bounds__(256) rmsnorm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                          const int* __restrict__ rows, A* __restrict__ y, int width, float eps) {
  __shared__ float red[40];
  const long long src = rows ? rows[blockIdx.x] : blockIdx.x;
  const float* xr = x + src * width;
  A* yr = y + (long long)blockIdx.x * width;
  float ss = 0.f;
  if ((width & 3) == 0) {
    const float4* x4 = reinterpret_cast<const float4*>(xr);
    const float4* w4 = reinterpret_cast<const float4*>(w);
    float4 keep[4];
    int n = 0;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = threadIdx.x + k * 256;
      if (i < width / 4) {
        keep[k] = x4[i];
        ss += keep[k].x * keep[k].x + keep[k].y * keep[k].y + keep[k].z * keep[k].z + keep[k].w * keep[k].w;
        n = k + 1;
      }
    }
    for (int i = threadIdx.x + 1024; i < width / 4; i += 256) {
      const float4 v = x4[i];
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    ss = block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / width + eps);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = threadIdx.x + k * 256;
      if (k < n) {
        const float4 g = w4[i];
        store4(yr + 4 * i, keep[k].x * r * g.x, keep[k].y * r * g.y, keep[k].z * r * g.z, keep[k].w * r * g.w);
      }
    }
    for (int i = threadIdx.x + 1024; i < width / 4; i += 256) {
      const float4 v = x4[i], g = w4[i];
      store4(yr + 4 * i, v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += 256) ss += xr[i] * xr[i];
    ss = block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / width + eps);
    for (int i = threadIdx.x; i < width; i += 256) yr[i] = from_f<A>(xr[i] * r * w[i]);
  }
}

// ------------------------------------------------------------------ per-head RMSNorm of a recurrence's read-out, with gate
// y[t, h * dv + c] = o / rms(o over the head) * w[c] * sigmoid(gate[t, h * dv + c]) * mul; one warp per (token, head).
template <typename A>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w,
                                                             const A* __restrict__ gate, long long gate_ld, float mul,
                                                             A* __restrict__ y, long long y_ld, long long items, int H, int dv,
                                                             float eps) {
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= items) return;
  const long long t = item / H;
  const int h = (int)(item % H);
  const float* oh = o + (t * H + h) * dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) ss += oh[c] * oh[c];
  ss = warp_sum(ss);
  const float r = mul / sqrtf(ss / dv + eps);
  const A* gr = gate ? gate + t * gate_ld + (long long)h * dv : nullptr;
  A* yr = y + t * y_ld + (long long)h * dv;
  for (int c = lane; c < dv; c += 32) {
    float v = oh[c] * r * w[c];
    if (gr) v *= sigmoid_f(to_f(gr[c]));
    yr[c] = from_f<A>(v);
  }
}

// ------------------------------------------------------------------ carried convolution inputs
// Position p of a sequence keeps its projected row in entry p % taps of its slot, so a step that reads positions
// p-1 .. p-taps+1 and writes p touches different entries.
template <typename A>
__global__ void conv_ring_kernel(const A* __restrict__ u, long long u_ld, A* __restrict__ ring, const RaggedView rv, int C, int taps) {
  const int seq = blockIdx.x, back = blockIdx.y;   // back: tokens before the last one of the portion
  const int len = rv.cu[seq + 1] - rv.cu[seq];
  if (back >= len) return;
  const int pos = rv.pos0[seq] + len - 1 - back;
  const A* src = u + (long long)(rv.cu[seq + 1] - 1 - back) * u_ld;
  A* dst = ring + ((long long)rv.slot[seq] * taps + pos % taps) * C;
  for (int i = threadIdx.x; i < C; i += blockDim.x) dst[i] = src[i];
}

// ------------------------------------------------------------------ attention operands: convolution, norm, rotation, cache append
struct QkvParams {
  const void* u;              // projected rows: q at column 0, k at H * d, v at H * d + G * d
  long long u_ld;
  const float* wconv;         // [taps, C], C = H d + G d + G dv
  void* ring;                 // [slots, taps, C]
  const float* qn; const float* kn;   // [d]
  const double* inv_freq;     // [rot / 2]
  const float* talk;          // [H, H] (mixed-query output only)
  float* q_out;               // [T, H, d] fp32, or null
  void* qmix_out;             // [T, H, G d] activation type, or null
  void* k_out; void* v_out;   // packed rows for the prompt kernels, or null
  long long k_ld, v_ld;       // row pitches; V of head j starts at column j * dvp
  int dvp;
  const int* kv_row;          // [T] packed row of each token (null: the token's own index)
  void* k_cache; void* v_cache;       // [entries, G, d] / [entries, G, dv]
  const int* cache_entry;     // [T], -1: not kept
  RaggedView rv;
  int T, H, G, d, dv, taps, rot;
  int write_ring;             // one token per sequence: this launch also stores the token's own ring entry
  float eps;
};

template <typename A>
__device__ __forceinline__ float conv_at(const QkvParams& p, const A* __restrict__ row, int ch, int pos, int pos0, const A* __restrict__ ring) {
  const int C = p.H * p.d + p.G * (p.d + p.dv);
  float acc = 0.f;
  for (int j = 0; j < p.taps; ++j) {
    const int b = p.taps - 1 - j;          // tokens back
    if (b > pos) continue;
    float x;
    if (pos - b >= pos0) x = to_f(row[ch - (long long)b * p.u_ld]);
    else x = to_f(ring[(long long)((pos - b) % p.taps) * C + ch]);
    acc = fmaf(p.wconv[(long long)j * C + ch], x, acc);
  }
  return acc;
}

template <typename A>
__global__ void __launch_bounds__(256) qkv_prep_kernel(const QkvParams p) {
  extern __shared__ float sm[];
  float* cs = sm;                    // [rot/2] cos
  float* sn = cs + p.rot / 2;        // [rot/2] sin
  float* sq = sn + p.rot / 2;        // [H, d] rotated queries (mixed-query output)
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int seq = p.rv.tok_seq[t], pos = p.rv.tok_pos[t], pos0 = p.rv.pos0[seq];
  const int C = p.H * p.d + p.G * (p.d + p.dv);
  const A* row = reinterpret_cast<const A*>(p.u) + (long long)t * p.u_ld;
  A* ring = reinterpret_cast<A*>(p.ring) + (long long)p.rv.slot[seq] * p.taps * C;
  const int entry = p.cache_entry[t];
  const long long krow = p.kv_row ? p.kv_row[t] : t;
  for (int i = threadIdx.x; i < p.rot / 2; i += blockDim.x) {
    double a = (double)pos * p.inv_freq[i];
    a -= 6.283185307179586476925286766559 * rint(a * 0.15915494309189533576888376337251);
    float s, c;
    sincosf((float)a, &s, &c);
    cs[i] = c;
    sn[i] = s;
  }
  __syncthreads();
  // one warp per query / key head; a lane owns the pairs (2i, 2i + 1) with i = lane, lane + 32, ..
  for (int hh = warp; hh < p.H + p.G; hh += nw) {
    const bool is_q = hh < p.H;
    const int ch0 = hh * p.d;
    const float* nw_ = is_q ? p.qn : p.kn;
    float va[QK_PAIRS], vb[QK_PAIRS];
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < QK_PAIRS; ++n) {
      const int i = lane + 32 * n;
      va[n] = vb[n] = 0.f;
      if (2 * i < p.d) {
        va[n] = conv_at<A>(p, row, ch0 + 2 * i, pos, pos0, ring);
        vb[n] = conv_at<A>(p, row, ch0 + 2 * i + 1, pos, pos0, ring);
        ss += va[n] * va[n] + vb[n] * vb[n];
      }
    }
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / p.d + p.eps);
#pragma unroll
    for (int n = 0; n < QK_PAIRS; ++n) {
      const int i = lane + 32 * n;
      if (2 * i >= p.d) continue;
      float a = va[n] * r * nw_[2 * i], b = vb[n] * r * nw_[2 * i + 1];
      if (2 * i < p.rot) {
        const float c = cs[i], s = sn[i];
        const float a2 = a * c - b * s, b2 = b * c + a * s;
        a = a2;
        b = b2;
      }
      if (is_q) {
        if (p.q_out) *reinterpret_cast<float2*>(p.q_out + ((long long)t * p.H + hh) * p.d + 2 * i) = make_float2(a, b);
        if (p.qmix_out) {
          sq[hh * p.d + 2 * i] = a;
          sq[hh * p.d + 2 * i + 1] = b;
        }
      } else {
        const int col = (hh - p.H) * p.d + 2 * i;
        if (p.k_out) store2(reinterpret_cast<A*>(p.k_out) + krow * p.k_ld + col, a, b);
        if (entry >= 0) store2(reinterpret_cast<A*>(p.k_cache) + (long long)entry * p.G * p.d + col, a, b);
      }
    }
  }
  const int vch0 = (p.H + p.G) * p.d;
  for (int c = threadIdx.x; c < p.G * p.dv; c += blockDim.x) {
    const A v = from_f<A>(conv_at<A>(p, row, vch0 + c, pos, pos0, ring));
    if (p.v_out) reinterpret_cast<A*>(p.v_out)[krow * p.v_ld + (c / p.dv) * p.dvp + c % p.dv] = v;
    if (entry >= 0) reinterpret_cast<A*>(p.v_cache)[(long long)entry * p.G * p.dv + c] = v;
  }
  if (p.write_ring && p.taps > 1 && p.rv.slot[seq] >= 0)
    for (int c = threadIdx.x; c < C; c += blockDim.x) ring[(long long)(pos % p.taps) * C + c] = row[c];
  if (p.qmix_out) {
    // The head mix is linear in the scores, so it is folded into the queries: mixed head h meets the concatenated key
    // row of all key heads with sum over the query heads g of key head j of talk[h, g] q_g in block j.
    __syncthreads();
    const int grp = p.H / p.G, Gd = p.G * p.d;
    A* out = reinterpret_cast<A*>(p.qmix_out) + (long long)t * p.H * Gd;
    for (int i = threadIdx.x; i < p.H * Gd / 2; i += blockDim.x) {
      const int h = (2 * i) / Gd, c = (2 * i) % Gd, j = c / p.d, e = c % p.d;
      float a = 0.f, b = 0.f;
      for (int g = 0; g < grp; ++g) {
        const float w = p.talk[h * p.H + j * grp + g];
        const float2 qv = *reinterpret_cast<const float2*>(&sq[(j * grp + g) * p.d + e]);
        a = fmaf(w, qv.x, a);
        b = fmaf(w, qv.y, b);
      }
      store2(out + 2 * i, a, b);
    }
  }
}

// ------------------------------------------------------------------ earlier keys of the current chunk: cache -> packed rows
template <typename A>
__global__ void kv_gather_kernel(const A* __restrict__ cache, const int* __restrict__ entry, const int* __restrict__ row,
                                 A* __restrict__ out, long long out_ld, int G, int w, int wp) {
  const A* src = cache + (long long)entry[blockIdx.x] * G * w;
  A* dst = out + (long long)row[blockIdx.x] * out_ld;
  for (int i = threadIdx.x; i < G * w; i += blockDim.x) dst[(i / w) * wp + i % w] = src[i];
}

}  // namespace sx
using namespace sx;


extern "C" int sx_embed_f32(const void* table, const int* ids, float* x, int T, int width, int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  SX_ACT_DISPATCH(f32, (embed_f32_kernel<A><<<T, 256, 0, st>>>((const A*)table, ids, x, width)));
  return last_rc();
}
extern "C" int sx_rmsnorm_f32(const float* x, const float* w, const int* rows, void* y, int T, int width, float eps, int f32,
                              cudaStream_t st) {
  if (T <= 0) return 0;
  SX_ACT_DISPATCH(f32, (rmsnorm_f32_kernel<A><<<T, 256, 0, st>>>(x, w, rows, (A*)y, width, eps)));
  return last_rc();
}
extern "C" int sx_head_norm_gate(const float* o, const float* w, const void* gate, long long gate_ld, float mul, void* y,
                                 long long y_ld, int T, int H, int dv, float eps, int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  const long long items = (long long)T * H;
  SX_ACT_DISPATCH(f32, (head_norm_gate_kernel<A><<<(unsigned)((items + 7) / 8), 256, 0, st>>>(
      o, w, (const A*)gate, gate_ld, mul, (A*)y, y_ld, items, H, dv, eps)));
  return last_rc();
}
extern "C" int sx_conv_ring(const void* u, long long u_ld, void* ring, const SxRagged* r, int C, int taps, int f32, cudaStream_t st) {
  if (r->n <= 0 || taps <= 1) return 0;
  const RaggedView rv = view(r);
  SX_ACT_DISPATCH(f32, (conv_ring_kernel<A><<<dim3(r->n, taps - 1), 256, 0, st>>>((const A*)u, u_ld, (A*)ring, rv, C, taps)));
  return last_rc();
}
extern "C" int sx_qkv_prep(const SxQkvArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (a->d % 2 || a->rot % 2 || a->rot > a->d || a->d > 64 * QK_PAIRS || a->G <= 0 || a->H % a->G) return -1;
  QkvParams p;
  p.u = a->u; p.u_ld = a->u_ld; p.wconv = a->wconv; p.ring = a->ring; p.qn = a->qn; p.kn = a->kn; p.inv_freq = a->inv_freq;
  p.talk = a->talk; p.q_out = a->q_out; p.qmix_out = a->qmix_out; p.k_out = a->k_out; p.v_out = a->v_out;
  p.k_ld = a->k_ld; p.v_ld = a->v_ld; p.dvp = a->dvp; p.kv_row = a->kv_row; p.k_cache = a->k_cache; p.v_cache = a->v_cache;
  p.cache_entry = a->cache_entry; p.rv = view(&a->ragged);
  p.T = a->T; p.H = a->H; p.G = a->G; p.d = a->d; p.dv = a->dv; p.taps = a->taps; p.rot = a->rot;
  p.write_ring = a->write_ring; p.eps = a->eps;
  const int smem = (a->rot + (a->qmix_out ? a->H * a->d : 0)) * 4;
  if (smem > 200 * 1024) return -2;
  SX_ACT_DISPATCH(a->f32, {
    static int set = 0;
    if (smem > 48 * 1024 && set < smem) {
      if (cudaFuncSetAttribute(qkv_prep_kernel<A>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -10;
      set = smem;
    }
    qkv_prep_kernel<A><<<a->T, 256, smem, st>>>(p);
  });
  return last_rc();
}
extern "C" int sx_kv_gather(const void* cache, const int* entry, const int* row, int n, void* out, long long out_ld, int G, int w,
                            int wp, int f32, cudaStream_t st) {
  if (n <= 0) return 0;
  SX_ACT_DISPATCH(f32, (kv_gather_kernel<A><<<n, 128, 0, st>>>((const A*)cache, entry, row, (A*)out, out_ld, G, w, wp)));
  return last_rc();
}
