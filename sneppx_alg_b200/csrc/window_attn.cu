// Sliding-window attention whose older keys are averages of whole blocks of tokens: operand preparation, block averages, the
// SIMT form for any head count and size (32-bit runs, and sizes the tensor-core kernels do not take), and the merge of key
// slices. A query at position p sees the tokens p - size + 1 .. p and, before them, floor((p - size + 1) / pool) averaged
// blocks, all in one softmax whose denominator also holds exp(sink) of the head.
// Values are rotated by their position before they are cached, outputs turned back by the query's position, so the weight of a
// value depends on its distance.
#include "window_attn.cuh"

namespace sx {

struct WinPrepParams {
  SxWinPrepArgs a;
  RaggedView rv;
};

__device__ __forceinline__ void turn_angle(double freq, int pos, float* c, float* s, bool exact) {
  double a = (double)pos * freq;
  a -= 6.283185307179586476925286766559 * rint(a * 0.15915494309189533576888376337251);
  if (exact) sincosf((float)a, s, c);
  else __sincosf((float)a, s, c);        // |a| <= pi: within 2^-21 there
}
// Places of pair m of n: halves (m, m + n) or neighbours (2 m, 2 m + 1).
__device__ __forceinline__ int2 pair_at(int m, int n, int interleaved) {
  return interleaved ? make_int2(2 * m, 2 * m + 1) : make_int2(m, m + n);
}

// Decoding: the block of p.pool positions that the row of sequence `seq` at `pos` completes becomes an average in the cache.
// All threads of the CTA that appended the row take part.
template <typename A>
__device__ __forceinline__ void win_pool_step(const SxWinPrepArgs& p, int seq, int pos) {
  if (!p.pool_entry) return;
  const int done = p.pool_entry[seq];
  if (done < 0) return;
  __syncthreads();                            // this row's entry is in the cache
  const int* table = p.block_table + (long long)seq * p.table_ld;
  const int first = pos - p.pool + 1, b0 = p.block_base[seq], G = p.G, d = p.d, dv = p.dv;
  for (int i = threadIdx.x; i < G * (d + dv); i += blockDim.x) {
    const bool is_v = i >= G * d;
    const int wd = is_v ? G * dv : G * d, c = is_v ? i - G * d : i;
    A* cache = reinterpret_cast<A*>(is_v ? p.v_cache : p.k_cache);
    float s = 0.f;
#pragma unroll 4
    for (int j = first; j <= pos; ++j)
      s += to_f(cache[((long long)table[j / p.block_size - b0] * p.block_size + j % p.block_size) * wd + c]);
    cache[(long long)done * wd + c] = from_f<A>(s / p.pool);
  }
}

// ------------------------------------------------------------------ operands: one CTA per row
template <typename A>
__global__ void __launch_bounds__(256) win_prep_kernel(const WinPrepParams P) {
  const SxWinPrepArgs& p = P.a;
  extern __shared__ __align__(16) float sm[];
  const int t = blockIdx.x, tid = threadIdx.x, seq = P.rv.tok_seq[t], pos = P.rv.tok_pos[t];
  if (P.rv.slot[seq] < 0) return;             // padding row of a captured launch
  const int d = p.d, dv = p.dv, nr = p.rot / 2, nv = dv / 2, H = p.H, G = p.G;
  float2* qc = reinterpret_cast<float2*>(sm); // [nr] cos, sin of the query / key angles, with their factor
  float2* vc = qc + nr;                       // [nv]
  for (int i = tid; i < nr + nv; i += 256) {
    float c, s;
    turn_angle(i < nr ? p.freq[i] : p.vfreq[i - nr], pos, &c, &s, sizeof(A) == 4);
    if (i < nr) {
      qc[i] = make_float2(c * p.rot_mul, s * p.rot_mul);
    } else {
      vc[i - nr] = make_float2(c, s);
      reinterpret_cast<float2*>(p.turn)[(long long)t * nv + i - nr] = make_float2(c, s);
    }
  }
  __syncthreads();
  const A* u = reinterpret_cast<const A*>(p.u) + (long long)t * p.u_ld;
  const int entry = p.cache_entry[t], krow = p.k_out ? (p.kv_row ? p.kv_row[t] : t) : 0;
  A* ko = reinterpret_cast<A*>(p.k_out) + (long long)krow * p.k_ld;
  A* vo = reinterpret_cast<A*>(p.v_out) + (long long)krow * p.v_ld;
  A* kc = reinterpret_cast<A*>(p.k_cache) + (long long)entry * G * d;
  A* vch = reinterpret_cast<A*>(p.v_cache) + (long long)entry * G * dv;
  auto in = [&](int col) { return to_f(u[col]) + (p.bias ? p.bias[col] : 0.f); };
  const int w = d - nr;                       // work items of a query or key head: pairs, then single entries
  for (int i = tid; i < (H + G) * w; i += 256) {
    const int h = i / w, e = i - h * w, base = h * d;
    int2 at;
    float a, b = 0.f;
    const bool pair = e < nr;
    if (pair) {
      at = pair_at(e, nr, p.interleaved);
      const float x = in(base + at.x), y = in(base + at.y);
      const float2 cs = qc[e];
      a = x * cs.x - y * cs.y;
      b = y * cs.x + x * cs.y;
    } else {
      at = make_int2(e + nr, 0);
      a = in(base + at.x);
    }
    if (h < H) {
      const float f = p.temp ? p.temp[h] : 1.f;
      if (p.q32) {
        float* q = p.q32 + ((long long)t * H + h) * d;
        q[at.x] = a * f;
        if (pair) q[at.y] = b * f;
      }
      if (p.q) {
        A* q = reinterpret_cast<A*>(p.q) + ((long long)t * H + h) * p.q_ld;
        q[at.x] = from_f<A>(a * f);
        if (pair) q[at.y] = from_f<A>(b * f);
      }
    } else {
      const int j = h - H;
      const A x = from_f<A>(a), y = from_f<A>(b);
      if (p.k_out) {
        ko[j * p.dp + at.x] = x;
        if (pair) ko[j * p.dp + at.y] = y;
      }
      if (entry >= 0) {
        kc[j * d + at.x] = x;
        if (pair) kc[j * d + at.y] = y;
      }
    }
  }
  for (int i = tid; i < G * nv; i += 256) {
    const int j = i / nv, e = i - j * nv;
    const int2 at = pair_at(e, nv, p.interleaved);
    const int base = (H + G) * d + j * dv;
    const float x = in(base + at.x), y = in(base + at.y);
    const float2 cs = vc[e];
    const A a = from_f<A>(x * cs.x - y * cs.y), b = from_f<A>(y * cs.x + x * cs.y);
    if (p.v_out) {
      vo[j * p.dvp + at.x] = a;
      vo[j * p.dvp + at.y] = b;
    }
    if (entry >= 0) {
      vch[j * dv + at.x] = a;
      vch[j * dv + at.y] = b;
    }
  }
  if (p.q && p.q_ld > d) {
    A* q = reinterpret_cast<A*>(p.q) + (long long)t * H * p.q_ld;
    const int pad = p.q_ld - d;
    for (int i = tid; i < H * pad; i += 256) q[(i / pad) * p.q_ld + d + i % pad] = from_f<A>(0.f);
  }
  win_pool_step<A>(p, seq, pos);
}

// ------------------------------------------------------------------ the same with 16-byte pieces (bf16, halves)
// One CTA: NT rows. A thread keeps its piece of the row (8 pairs, or 8 entries that pass unchanged) for all of them, so that
// biases are read once and the loads of all rows are in flight together.
template <int NT>
__global__ void __launch_bounds__(256, 3) win_prep_vec_kernel(const WinPrepParams P) {
  using bf = __nv_bfloat16;
  const SxWinPrepArgs& p = P.a;
  extern __shared__ __align__(16) float sm[];
  const int t0 = blockIdx.x * NT, tid = threadIdx.x, n = blockDim.x, nt = min(NT, p.T - t0);
  const int d = p.d, dv = p.dv, nr = p.rot / 2, nv = dv / 2, H = p.H, G = p.G;
  float2* cs = reinterpret_cast<float2*>(sm); // [NT][nr + nv] cos, sin; those of queries and keys with their factor
  const int wq = nr / 8 + (d - p.rot) / 8, wv = nv / 8, items = (H + G) * wq + G * wv;
  bf16x8 x[NT], y[NT];
  bool is_v, pair;
  int h, a0, a1, base;                        // head, its two pieces' columns, its first column in the row
  auto load = [&](int i) {
    is_v = i >= (H + G) * wq;
    const int j = is_v ? i - (H + G) * wq : i, w = is_v ? wv : wq, e = j % w;
    h = j / w;
    pair = is_v || e < nr / 8;
    a0 = pair ? e * 8 : p.rot + (e - nr / 8) * 8;
    a1 = a0 + (is_v ? nv : nr);
    base = is_v ? (H + G) * d + h * dv : h * d;
    const bf* u = reinterpret_cast<const bf*>(p.u) + (long long)t0 * p.u_ld + base;
#pragma unroll
    for (int t = 0; t < NT; ++t)
      if (t < nt) {
        x[t] = ld8(u + t * p.u_ld + a0);
        y[t] = ld8(u + t * p.u_ld + (pair ? a1 : a0));
      }
  };
  if (tid < items) load(tid);                 // arrives while the angles are worked out
#pragma unroll
  for (int t = 0; t < NT; ++t) {
    if (t >= nt) break;
    const int pos = P.rv.tok_pos[t0 + t];
    for (int e = tid; e < nr + nv; e += n) {
      float c, s;
      turn_angle(e < nr ? p.freq[e] : p.vfreq[e - nr], pos, &c, &s, false);
      cs[t * (nr + nv) + e] = e < nr ? make_float2(c * p.rot_mul, s * p.rot_mul) : make_float2(c, s);
      if (e >= nr) reinterpret_cast<float2*>(p.turn)[(long long)(t0 + t) * nv + e - nr] = make_float2(c, s);
    }
  }
  __syncthreads();
  for (int i = tid; i < items; i += n) {
    if (i != tid) load(i);
    float bx[8], by[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      bx[k] = p.bias ? p.bias[base + a0 + k] : 0.f;
      by[k] = p.bias && pair ? p.bias[base + a1 + k] : 0.f;
    }
    const float f = !is_v && h < H && p.temp ? p.temp[h] : 1.f;
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      if (t >= nt) break;
      const int row = t0 + t;
      if (P.rv.slot[P.rv.tok_seq[row]] < 0) continue;            // padding row of a captured launch
      float a[8], b[8];
      unpack8(x[t], a);
      unpack8(y[t], b);
      const float2* c = cs + t * (nr + nv) + (is_v ? nr : 0) + a0;
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float u0 = a[k] + bx[k], u1 = b[k] + by[k];
        if (pair) {
          const float2 q = c[k];
          a[k] = (u0 * q.x - u1 * q.y) * f;
          b[k] = (u1 * q.x + u0 * q.y) * f;
        } else {
          a[k] = u0 * f;
        }
      }
      const bf16x8 oa = pack8(a), ob = pack8(b);
      auto put = [&](bf* dst) {
        st8(dst + a0, oa);
        if (pair) st8(dst + a1, ob);
      };
      if (!is_v && h < H) {
        put(reinterpret_cast<bf*>(p.q) + ((long long)row * H + h) * p.q_ld);
      } else {
        const int g = is_v ? h : h - H, entry = p.cache_entry[row];
        bf* out = reinterpret_cast<bf*>(is_v ? p.v_out : p.k_out);
        if (out) put(out + (long long)(p.kv_row ? p.kv_row[row] : row) * (is_v ? p.v_ld : p.k_ld) + g * (is_v ? p.dvp : p.dp));
        if (entry >= 0) put(reinterpret_cast<bf*>(is_v ? p.v_cache : p.k_cache) + ((long long)entry * G + g) * (is_v ? dv : d));
      }
    }
  }
  if (p.q_ld > d) {
    const int pad = (p.q_ld - d) / 8;
    for (int i = tid; i < nt * H * pad; i += n)
      *reinterpret_cast<uint4*>(reinterpret_cast<bf*>(p.q) + ((long long)t0 * H + i / pad) * p.q_ld + d + i % pad * 8) = make_uint4(0, 0, 0, 0);
  }
  if (NT == 1 && P.rv.slot[P.rv.tok_seq[t0]] >= 0) win_pool_step<bf>(p, P.rv.tok_seq[t0], P.rv.tok_pos[t0]);
}

// ------------------------------------------------------------------ averages of the blocks that a prompt batch completes
template <typename A>
__global__ void __launch_bounds__(256) pool_blocks_kernel(A* __restrict__ rows, long long ld, int wp, A* __restrict__ cache, int G, int w,
                                                          const int* __restrict__ src, const int* __restrict__ row,
                                                          const int* __restrict__ entry, int pool) {
  const int b = blockIdx.x;
  const A* x = rows + (long long)src[b] * ld;
  A* out = rows + (long long)row[b] * ld;
  A* ce = cache + (long long)entry[b] * G * w;
  for (int i = threadIdx.x; i < G * w; i += 256) {
    const int c = i / w * wp + i % w;
    float s = 0.f;
    for (int j = 0; j < pool; ++j) s += to_f(x[j * ld + c]);
    const A m = from_f<A>(s / pool);
    out[c] = m;
    ce[i] = m;
  }
}

// ------------------------------------------------------------------ SIMT form: one CTA per (row, key head, key slice)
constexpr int WA_KT = 32;     // keys per tile

template <typename A, bool PAGED>
__global__ void __launch_bounds__(128) win_attn_kernel(const WinParams P) {
  const SxWinAttnArgs& p = P.a;
  extern __shared__ __align__(16) float sm[];
  const int H = p.H, G = p.G, d = p.d, dv = p.dv, grp = H / G;
  float* sq = sm;                       // [grp, d]
  float* pr = sq + grp * d;             // [grp, KT]
  float* so = pr + grp * WA_KT;         // [grp, dv]
  float* sm_m = so + grp * dv;          // [grp]
  float* sm_l = sm_m + grp;
  float* sm_c = sm_l + grp;
  const int t = blockIdx.x, g = blockIdx.y, split = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = P.rv.tok_seq[t], pos = P.rv.tok_pos[t];
  if (P.rv.slot[seq] < 0) return;
  const WinKeys keys = win_keys(pos, p.size, p.pool);
  const int n = keys.blocks + keys.tokens, per = (n + p.splits - 1) / p.splits;
  const int lo = min(n, split * per), hi = min(n, lo + per);
  for (int i = tid; i < grp * d; i += 128) sq[i] = p.q32[((long long)t * H + g * grp) * d + i] * p.scale;
  for (int i = tid; i < grp * dv; i += 128) so[i] = 0.f;
  for (int i = tid; i < grp; i += 128) {
    sm_m[i] = -INFINITY;
    sm_l[i] = 0.f;
  }
  const A* K = reinterpret_cast<const A*>(p.k) + g * p.dp;
  const A* V = reinterpret_cast<const A*>(p.v) + g * p.dvp;
  auto row_of = [&](int i) -> long long {
    if constexpr (PAGED) return win_entry(P, seq, keys, i);
    else return i < keys.blocks ? (long long)p.pool_base[seq] + i : (long long)p.kv_base[seq] + keys.first + i - keys.blocks;
  };
  for (int j0 = lo; j0 < hi; j0 += WA_KT) {
    const int nk = min(WA_KT, hi - j0);
    __syncthreads();
    for (int i = tid; i < grp * WA_KT; i += 128) {
      const int h = i / WA_KT, j = i % WA_KT;
      float s = -INFINITY;
      if (j < nk) {
        const A* k = K + row_of(j0 + j) * p.k_ld;
        s = 0.f;
        for (int c = 0; c < d; ++c) s = fmaf(sq[h * d + c], to_f(k[c]), s);
      }
      pr[i] = s;
    }
    __syncthreads();
    for (int h = warp; h < grp; h += 4) {
      const float s = pr[h * WA_KT + lane];
      const float m_old = sm_m[h], m = fmaxf(m_old, warp_max(s));
      const float e = expf(s - m);
      const float l = warp_sum(e);
      pr[h * WA_KT + lane] = e;
      if (lane == 0) {
        const float c = expf(m_old - m);
        sm_c[h] = c;
        sm_m[h] = m;
        sm_l[h] = sm_l[h] * c + l;
      }
    }
    __syncthreads();
    for (int i = tid; i < grp * dv; i += 128) {
      const int h = i / dv, c = i % dv;
      float acc = so[i] * sm_c[h];
      for (int j = 0; j < nk; ++j) acc = fmaf(pr[h * WA_KT + j], to_f(V[row_of(j0 + j) * p.v_ld + c]), acc);
      so[i] = acc;
    }
  }
  __syncthreads();
  if (p.part) {
    float* part = p.part + (((long long)t * p.splits + split) * H + g * grp) * (dv + 2);
    for (int i = tid; i < grp * dv; i += 128) part[(i / dv) * (dv + 2) + 2 + i % dv] = so[i];
    for (int h = tid; h < grp; h += 128) {
      part[h * (dv + 2)] = sm_m[h];
      part[h * (dv + 2) + 1] = sm_l[h];
    }
    return;
  }
  const int nv = dv / 2;
  for (int i = tid; i < grp * nv; i += 128) {
    const int hl = i / nv, e = i - hl * nv, h = g * grp + hl;
    const float m = fmaxf(sm_m[hl], p.sink[h]), f = expf(sm_m[hl] - m);
    const float inv = f / (sm_l[hl] * f + expf(p.sink[h] - m));
    const int2 at = pair_at(e, nv, p.interleaved);
    win_store<A>(P, t, h, e, at, so[hl * dv + at.x] * inv, so[hl * dv + at.y] * inv);
  }
}

// ------------------------------------------------------------------ merge of key slices
template <typename A>
__global__ void __launch_bounds__(64) win_merge_kernel(const WinParams P) {
  const SxWinAttnArgs& p = P.a;
  const int h = blockIdx.x, t = blockIdx.y, dv = p.dv, nv = dv / 2;
  if (P.rv.slot[P.rv.tok_seq[t]] < 0) return;
  const float* part = p.part + ((long long)t * p.splits * p.H + h) * (dv + 2);
  const long long step = (long long)p.H * (dv + 2);
  float m = p.sink[h];
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, part[s * step]);
  float l = expf(p.sink[h] - m);
  for (int s = 0; s < p.splits; ++s) l += part[s * step + 1] * expf(part[s * step] - m);
  const float inv = 1.f / l;
  for (int e = threadIdx.x; e < nv; e += 64) {
    const int2 at = pair_at(e, nv, p.interleaved);
    float a = 0.f, b = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float f = expf(part[s * step] - m);
      a = fmaf(part[s * step + 2 + at.x], f, a);
      b = fmaf(part[s * step + 2 + at.y], f, b);
    }
    win_store<A>(P, t, h, e, at, a * inv, b * inv);
  }
}

}  // namespace sx
using namespace sx;

extern "C" int sx_win_prep(const SxWinPrepArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (a->d <= 0 || a->dv <= 0 || a->dv % 2 || a->rot % 2 || a->rot > a->d || a->G <= 0 || a->H % a->G) return -1;
  const WinPrepParams p{*a, view(&a->ragged)};
  const int smem = (a->rot + a->dv) * 4;
  if (smem > 12 * 1024) return -2;
  const auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  const bool vec = !a->f32 && !a->interleaved && a->q && !a->q32 && a->rot % 16 == 0 && a->d % 8 == 0 && a->dv % 16 == 0 && a->u_ld % 8 == 0 &&
                   a->q_ld % 8 == 0 && al(a->u) && al(a->q) && al(a->k_cache) && al(a->v_cache) &&
                   (!a->k_out || (al(a->k_out) && al(a->v_out) && a->k_ld % 8 == 0 && a->v_ld % 8 == 0 && a->dp % 8 == 0 && a->dvp % 8 == 0));
  if (vec) {
    const int items = (a->H + a->G) * (a->d - a->rot / 2) / 8 + a->G * a->dv / 16;
    const int threads = items >= 256 ? 256 : items <= 32 ? 32 : (items + 31) / 32 * 32;
    if (a->T >= 4 * 148 && !a->pool_entry) win_prep_vec_kernel<4><<<(a->T + 3) / 4, threads, 4 * smem, st>>>(p);
    else win_prep_vec_kernel<1><<<a->T, threads, smem, st>>>(p);
    return last_rc();
  }
  SX_ACT_DISPATCH(a->f32, (win_prep_kernel<A><<<a->T, 256, smem, st>>>(p)));
  return last_rc();
}

extern "C" int sx_pool_blocks(void* rows, long long ld, int wp, void* cache, int G, int w, const int* src, const int* row, const int* entry,
                              int n, int pool, int f32, cudaStream_t st) {
  if (n <= 0) return 0;
  if (pool <= 0) return -1;
  SX_ACT_DISPATCH(f32, (pool_blocks_kernel<A><<<n, 256, 0, st>>>((A*)rows, ld, wp, (A*)cache, G, w, src, row, entry, pool)));
  return last_rc();
}

extern "C" int sx_win_merge(const SxWinAttnArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  const WinParams p{*a, view(&a->ragged)};
  SX_ACT_DISPATCH(a->f32, (win_merge_kernel<A><<<dim3(a->H, a->T), 64, 0, st>>>(p)));
  return last_rc();
}

template <typename A>
static int launch_win(const WinParams& p, cudaStream_t st) {
  const SxWinAttnArgs& a = p.a;
  const int grp = a.H / a.G, smem = grp * (a.d + WA_KT + a.dv + 3) * 4;
  if (smem > 227 * 1024) return -2;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(win_attn_kernel<A, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(win_attn_kernel<A, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess)
      return -10;
    set = true;
  }
  const dim3 grid(a.T, a.G, a.splits);
  if (a.block_table) win_attn_kernel<A, true><<<grid, 128, smem, st>>>(p);
  else win_attn_kernel<A, false><<<grid, 128, smem, st>>>(p);
  return last_rc();
}

extern "C" int sx_win_attn(const SxWinAttnArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (a->G <= 0 || a->H % a->G || a->dv % 2 || a->size <= 0 || a->pool <= 0 || a->splits < 1 || (a->splits > 1 && !a->part)) return -1;
  const WinParams p{*a, view(&a->ragged)};
  int rc = 0;
  SX_ACT_DISPATCH(a->f32, { rc = launch_win<A>(p, st); });
  return rc == 0 && a->part ? sx_win_merge(a, st) : rc;
}
