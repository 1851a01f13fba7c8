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
__global__ void embed_f32_kernel(const A* __restrict__ table, const int* __restrict__ ids, float* __restrict__ x, int width, float scale) {
  const A* src = table + (long long)ids[blockIdx.x] * width;
  float* dst = x + (long long)blockIdx.x * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = to_f(src[i]) * scale;
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

// ------------------------------------------------------------------ layer norm of fp32 rows
// y = (x - mean) / sqrt(mean of squared deviations + eps) * w + b. Rows as in the RMSNorm; up to 4096 entries of a row stay in
// registers between the passes.
template <typename A>
__global__ void __launch_bounds__(256) layernorm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                            const float* __restrict__ b, const int* __restrict__ rows,
                                                            A* __restrict__ y, int width, float eps) {
  __shared__ float red[40];
  const long long src = rows ? rows[blockIdx.x] : blockIdx.x;
  const float* xr = x + src * width;
  A* yr = y + (long long)blockIdx.x * width;
  if ((width & 3) == 0) {
    const float4* x4 = reinterpret_cast<const float4*>(xr);
    const float4* w4 = reinterpret_cast<const float4*>(w);
    const float4* b4 = reinterpret_cast<const float4*>(b);
    const int n4 = width / 4;
    float4 keep[4];
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = threadIdx.x + k * 256;
      keep[k] = i < n4 ? x4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
      s += (keep[k].x + keep[k].y) + (keep[k].z + keep[k].w);
    }
    for (int i = threadIdx.x + 1024; i < n4; i += 256) {
      const float4 v = x4[i];
      s += (v.x + v.y) + (v.z + v.w);
    }
    const float m = block_sum(s, red) / width;
    float ss = 0.f;
    auto dev = [&](const float4& v) {
      const float a = v.x - m, c = v.y - m, d = v.z - m, e = v.w - m;
      ss += (a * a + c * c) + (d * d + e * e);
    };
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (threadIdx.x + k * 256 < n4) dev(keep[k]);
    for (int i = threadIdx.x + 1024; i < n4; i += 256) dev(x4[i]);
    const float r = 1.f / sqrtf(block_sum(ss, red) / width + eps);
    auto put = [&](int i, const float4& v) {
      const float4 g = w4[i], o = b4[i];
      store4(yr + 4 * i, fmaf((v.x - m) * r, g.x, o.x), fmaf((v.y - m) * r, g.y, o.y), fmaf((v.z - m) * r, g.z, o.z),
             fmaf((v.w - m) * r, g.w, o.w));
    };
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (threadIdx.x + k * 256 < n4) put(threadIdx.x + k * 256, keep[k]);
    for (int i = threadIdx.x + 1024; i < n4; i += 256) put(i, x4[i]);
  } else {
    float s = 0.f, ss = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) s += xr[i];
    const float m = block_sum(s, red) / width;
    for (int i = threadIdx.x; i < width; i += 256) ss += (xr[i] - m) * (xr[i] - m);
    const float r = 1.f / sqrtf(block_sum(ss, red) / width + eps);
    for (int i = threadIdx.x; i < width; i += 256) yr[i] = from_f<A>(fmaf((xr[i] - m) * r, w[i], b[i]));
  }
}

// ------------------------------------------------------------------ RMSNorm of equal parts of activation rows, in place
// One CTA per (row, part). VEC: parts, pitch and base allow 16-byte pieces; up to 4 pieces per thread stay in registers.
template <typename A, bool VEC>
__global__ void __launch_bounds__(256) part_rmsnorm_kernel(A* __restrict__ y, long long ld, const float* __restrict__ w, int part, float eps) {
  __shared__ float red[40];
  A* yr = y + (long long)blockIdx.x * ld + (long long)blockIdx.y * part;
  const float* wr = w + (long long)blockIdx.y * part;
  const int n = blockDim.x;
  float ss = 0.f;
  if constexpr (VEC) {
    constexpr int E = 16 / sizeof(A);
    const int pieces = part / E;
    uint4 keep[4];
    auto sum = [&](const uint4& v) {
      const A* a = reinterpret_cast<const A*>(&v);
#pragma unroll
      for (int e = 0; e < E; ++e) ss = fmaf(to_f(a[e]), to_f(a[e]), ss);
    };
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = threadIdx.x + k * n;
      if (i < pieces) {
        keep[k] = reinterpret_cast<const uint4*>(yr)[i];
        sum(keep[k]);
      }
    }
    for (int i = threadIdx.x + 4 * n; i < pieces; i += n) sum(reinterpret_cast<const uint4*>(yr)[i]);
    const float r = 1.f / sqrtf(block_sum(ss, red) / part + eps);
    auto put = [&](int i, const uint4& v) {
      const A* a = reinterpret_cast<const A*>(&v);
#pragma unroll
      for (int e = 0; e < E; e += 4) {
        const float4 g = *reinterpret_cast<const float4*>(wr + i * E + e);
        store4(yr + i * E + e, to_f(a[e]) * r * g.x, to_f(a[e + 1]) * r * g.y, to_f(a[e + 2]) * r * g.z, to_f(a[e + 3]) * r * g.w);
      }
    };
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (threadIdx.x + k * n < pieces) put(threadIdx.x + k * n, keep[k]);
    for (int i = threadIdx.x + 4 * n; i < pieces; i += n) {
      const uint4 v = reinterpret_cast<const uint4*>(yr)[i];
      put(i, v);
    }
  } else {
    for (int i = threadIdx.x; i < part; i += n) ss = fmaf(to_f(yr[i]), to_f(yr[i]), ss);
    const float r = 1.f / sqrtf(block_sum(ss, red) / part + eps);
    for (int i = threadIdx.x; i < part; i += n) yr[i] = from_f<A>(to_f(yr[i]) * r * wr[i]);
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
  const A* gr = gate ? gate + t * gate_ld + (long long)h * dv : nullptr;
  A* yr = y + t * y_ld + (long long)h * dv;
  float ss = 0.f;
  if (dv == 128) {     // one 16-byte piece per lane
    const float4 v = *reinterpret_cast<const float4*>(oh + lane * 4);
    ss = warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w);
    const float r = mul / sqrtf(ss / dv + eps);
    const float4 g = *reinterpret_cast<const float4*>(w + lane * 4);
    float out[4] = {v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (gr) out[i] *= sigmoid_f(to_f(gr[lane * 4 + i]));
#pragma unroll
    for (int i = 0; i < 4; i += 2) store2(yr + lane * 4 + i, out[i], out[i + 1]);
    return;
  }
  for (int c = lane; c < dv; c += 32) ss += oh[c] * oh[c];
  ss = warp_sum(ss);
  const float r = mul / sqrtf(ss / dv + eps);
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
  void* qmix_out;             // [T, H, qmix_ld] activation type, or null
  int qmix_ld;
  void* k_out; void* v_out;   // packed rows for the prompt kernels, or null
  long long k_ld, v_ld;       // row pitches; V of head j starts at column j * dvp
  int dvp;
  const int* kv_row;          // [T] packed row of each token (null: the token's own index)
  void* k_cache; void* v_cache;       // [entries, G, d] / [entries, G, dv]
  const int* cache_entry;     // [T], -1: not kept
  RaggedView rv;
  ChunkView cv;
  int T, H, G, d, dv, taps, rot;
  float eps;
};

// One CTA: NT rows of one portion (a chunk of a prompt, or the one row of a decode step) for one key head with its query
// heads and value head. A thread walks a channel through the rows; heads are then normed and rotated in shared memory.
template <typename A, int NT, int MT>
__global__ void __launch_bounds__(256, MT <= 4 ? 3 : 1) qkv_prep_kernel(const QkvParams p) {
  extern __shared__ __align__(16) float sm[];
  const int grp = p.H / p.G, nh = grp + 1, d = p.d, j = blockIdx.y;
  float* cs = sm;                    // [NT, rot/2] cos
  float* sn = cs + NT * (p.rot / 2); // [NT, rot/2] sin
  float* sh = sn + NT * (p.rot / 2); // [NT, grp + 1, d] query heads of the group, then the key head
  float* st = sh + NT * nh * d;      // [H, grp] head mix towards this group's queries
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = NT == 1 ? blockIdx.x : p.cv.seq[blockIdx.x], s0 = NT == 1 ? 0 : p.cv.start[blockIdx.x];
  const int slot = p.rv.slot[seq];
  if (slot < 0) return;              // padding row of a captured launch
  const int row0 = p.rv.cu[seq] + s0, nt = NT == 1 ? 1 : min(NT, p.rv.cu[seq + 1] - row0), pos = p.rv.pos0[seq] + s0;
  const int C = p.H * d + p.G * (d + p.dv);
  const A* u = reinterpret_cast<const A*>(p.u) + (long long)row0 * p.u_ld;
  A* ring = reinterpret_cast<A*>(p.ring) + (long long)slot * p.taps * C;
  for (int i = tid; i < NT * (p.rot / 2); i += 256) {
    const int t = i / (p.rot / 2);
    double a = (double)(pos + t) * p.inv_freq[i - t * (p.rot / 2)];
    a -= 6.283185307179586476925286766559 * rint(a * 0.15915494309189533576888376337251);
    float s, c;
    if (sizeof(A) == 4) sincosf((float)a, &s, &c);
    else __sincosf((float)a, &s, &c);       // |a| <= pi: within 2^-21 there
    cs[i] = c;
    sn[i] = s;
  }
  if (p.qmix_out)
    for (int i = tid; i < p.H * grp; i += 256) st[i] = p.talk[(i / grp) * p.H + j * grp + i % grp];
  const int nqk = nh * d;
  for (int i = tid; i < nqk + p.dv; i += 256) {
    const bool is_v = i >= nqk;
    const int ch = is_v ? (p.H + p.G) * d + j * p.dv + i - nqk : (i < grp * d ? j * grp * d + i : (p.H + j) * d + i - grp * d);
    float y[NT];
    conv_walk<A, NT, MT>(u, p.u_ld, p.wconv, p.taps, C, ch, ring, pos, s0, nt, y);
    if (NT == 1 && p.taps > 1) ring[(long long)(pos % p.taps) * C + ch] = u[ch];   // not an entry that this step reads
    if (is_v) {
      const int c = i - nqk;
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        if (t >= nt) continue;
        const A v = from_f<A>(y[t]);
        if (p.v_out) reinterpret_cast<A*>(p.v_out)[(long long)p.kv_row[row0 + t] * p.v_ld + j * p.dvp + c] = v;
        const int entry = p.cache_entry[row0 + t];
        if (entry >= 0) reinterpret_cast<A*>(p.v_cache)[((long long)entry * p.G + j) * p.dv + c] = v;
      }
    } else {
#pragma unroll
      for (int t = 0; t < NT; ++t) sh[t * nqk + i] = y[t];
    }
  }
  __syncthreads();
  // one warp per head row: RMS norm and rotation of the pairs (2i, 2i + 1)
  for (int t = 0, hh = warp; t < nt; hh += 8) {
    while (hh >= nh) {
      hh -= nh;
      ++t;
    }
    if (t >= nt) break;
    float* x = sh + t * nqk + hh * d;
    float ss = 0.f;
    for (int i = lane; i < d / 2; i += 32) {
      const float2 v = *reinterpret_cast<const float2*>(x + 2 * i);
      ss += v.x * v.x + v.y * v.y;
    }
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / d + p.eps);
    const bool is_q = hh < grp;
    const float* w = is_q ? p.qn : p.kn;
    const long long krow = !is_q && p.k_out ? p.kv_row[row0 + t] : 0;
    const int entry = is_q ? -1 : p.cache_entry[row0 + t];
    for (int i = lane; i < d / 2; i += 32) {
      float2 v = *reinterpret_cast<const float2*>(x + 2 * i);
      v.x *= r * w[2 * i];
      v.y *= r * w[2 * i + 1];
      if (2 * i < p.rot) {
        const float c = cs[t * (p.rot / 2) + i], s = sn[t * (p.rot / 2) + i];
        v = make_float2(v.x * c - v.y * s, v.y * c + v.x * s);
      }
      if (is_q) {
        if (p.q_out) *reinterpret_cast<float2*>(p.q_out + ((long long)(row0 + t) * p.H + j * grp + hh) * d + 2 * i) = v;
        if (p.qmix_out) *reinterpret_cast<float2*>(x + 2 * i) = v;
      } else {
        const int col = j * d + 2 * i;
        if (p.k_out) store2(reinterpret_cast<A*>(p.k_out) + krow * p.k_ld + col, v.x, v.y);
        if (entry >= 0) store2(reinterpret_cast<A*>(p.k_cache) + (long long)entry * p.G * d + col, v.x, v.y);
      }
    }
  }
  if (!p.qmix_out) return;
  // The head mix is linear in the scores, so it is folded into the queries: mixed head h meets the concatenated key row of
  // all key heads with sum over the query heads g of key head j of talk[h, g] q_g in block j. This CTA writes block j.
  __syncthreads();
  A* out = reinterpret_cast<A*>(p.qmix_out) + (long long)row0 * p.H * p.qmix_ld;
  const int half = d / 2;
  if (NT >= 4 && grp == 4 && half <= 256 && 256 % half == 0) {
    // a thread keeps one pair of channels of up to four tokens: the mix weights of a head are read once for all of them
    const int e = tid % half, step = 256 / half;
    for (int t0 = tid / half; t0 < nt; t0 += 4 * step) {
      float2 q[4][4];
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          const int t = t0 + x * step;
          q[x][g] = t < nt ? *reinterpret_cast<const float2*>(sh + t * nqk + g * d + 2 * e) : make_float2(0.f, 0.f);
        }
      A* o = out + (long long)t0 * p.H * p.qmix_ld + j * d + 2 * e;
      const long long tstep = (long long)step * p.H * p.qmix_ld;
      const bool all = t0 + 3 * step < nt;
#pragma unroll 2
      for (int h = 0; h < p.H; ++h, o += p.qmix_ld) {
        const float w0 = st[h * 4], w1 = st[h * 4 + 1], w2 = st[h * 4 + 2], w3 = st[h * 4 + 3];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float a = fmaf(w0, q[x][0].x, fmaf(w1, q[x][1].x, fmaf(w2, q[x][2].x, w3 * q[x][3].x)));
          const float b = fmaf(w0, q[x][0].y, fmaf(w1, q[x][1].y, fmaf(w2, q[x][2].y, w3 * q[x][3].y)));
          if (all || t0 + x * step < nt) store2(o + x * tstep, a, b);
        }
      }
    }
  } else
  for (int i = tid; i < nt * half; i += 256) {
    const int t = i / half, e = i % half;
    const float* x = sh + t * nqk + 2 * e;
    A* o = out + (long long)t * p.H * p.qmix_ld + j * d + 2 * e;
    if (grp <= 8) {
      float2 q[8];
#pragma unroll
      for (int g = 0; g < 8; ++g) q[g] = g < grp ? *reinterpret_cast<const float2*>(x + g * d) : make_float2(0.f, 0.f);
      for (int h = 0; h < p.H; ++h) {
        float a = 0.f, b = 0.f;
#pragma unroll
        for (int g = 0; g < 8; ++g)
          if (g < grp) {
            const float w = st[h * grp + g];
            a = fmaf(w, q[g].x, a);
            b = fmaf(w, q[g].y, b);
          }
        store2(o + (long long)h * p.qmix_ld, a, b);
      }
    } else {
      for (int h = 0; h < p.H; ++h) {
        float a = 0.f, b = 0.f;
        for (int g = 0; g < grp; ++g) {
          const float w = st[h * grp + g];
          const float2 q = *reinterpret_cast<const float2*>(x + g * d);
          a = fmaf(w, q.x, a);
          b = fmaf(w, q.y, b);
        }
        store2(o + (long long)h * p.qmix_ld, a, b);
      }
    }
  }
  if (j == 0) {
    const int pad = p.qmix_ld - p.G * d;
    for (int i = tid; i < nt * p.H * pad; i += 256) out[(long long)(i / pad) * p.qmix_ld + p.G * d + i % pad] = from_f<A>(0.f);
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


extern "C" int sx_embed_f32(const void* table, const int* ids, float* x, int T, int width, float scale, int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  SX_ACT_DISPATCH(f32, (embed_f32_kernel<A><<<T, 256, 0, st>>>((const A*)table, ids, x, width, scale)));
  return last_rc();
}
extern "C" int sx_rmsnorm_f32(const float* x, const float* w, const int* rows, void* y, int T, int width, float eps, int f32,
                              cudaStream_t st) {
  if (T <= 0) return 0;
  SX_ACT_DISPATCH(f32, (rmsnorm_f32_kernel<A><<<T, 256, 0, st>>>(x, w, rows, (A*)y, width, eps)));
  return last_rc();
}
extern "C" int sx_layernorm_f32(const float* x, const float* w, const float* b, const int* rows, void* y, int T, int width, float eps,
                                int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  SX_ACT_DISPATCH(f32, (layernorm_f32_kernel<A><<<T, 256, 0, st>>>(x, w, b, rows, (A*)y, width, eps)));
  return last_rc();
}
extern "C" int sx_part_rmsnorm(void* y, long long ld, const float* w, int T, int width, int parts, float eps, int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (parts <= 0 || parts > 65535 || width % parts) return -1;
  const int part = width / parts, E = f32 ? 4 : 8;
  const bool vec = part % E == 0 && ld % E == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  const int threads = part >= 2048 ? 256 : part >= 512 ? 128 : 32;
  const dim3 grid(T, parts);
  SX_ACT_DISPATCH(f32, {
    if (vec) part_rmsnorm_kernel<A, true><<<grid, threads, 0, st>>>((A*)y, ld, w, part, eps);
    else part_rmsnorm_kernel<A, false><<<grid, threads, 0, st>>>((A*)y, ld, w, part, eps);
  });
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
template <typename A, int NT, int MT>
static int launch_qkv(const QkvParams& p, int ctas, cudaStream_t st) {
  const int grp = p.H / p.G;
  const int smem = (NT * p.rot + NT * (grp + 1) * p.d + p.H * grp) * 4;
  static int set = 48 * 1024;
  if (smem > 227 * 1024) return -2;
  if (smem > set) {
    if (cudaFuncSetAttribute(qkv_prep_kernel<A, NT, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -10;
    set = smem;
  }
  qkv_prep_kernel<A, NT, MT><<<dim3(ctas, p.G), 256, smem, st>>>(p);
  return last_rc();
}
extern "C" int sx_qkv_prep(const SxQkvArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (a->d % 2 || a->rot % 2 || a->rot > a->d || a->G <= 0 || a->H % a->G || a->taps < 1 || a->taps > 8) return -1;
  QkvParams p;
  p.u = a->u; p.u_ld = a->u_ld; p.wconv = a->wconv; p.ring = a->ring; p.qn = a->qn; p.kn = a->kn; p.inv_freq = a->inv_freq;
  p.talk = a->talk; p.q_out = a->q_out; p.qmix_out = a->qmix_out; p.qmix_ld = a->qmix_ld; p.k_out = a->k_out; p.v_out = a->v_out;
  p.k_ld = a->k_ld; p.v_ld = a->v_ld; p.dvp = a->dvp; p.kv_row = a->kv_row; p.k_cache = a->k_cache; p.v_cache = a->v_cache;
  p.cache_entry = a->cache_entry; p.rv = view(&a->ragged); p.cv = chunks(&a->chunks);
  p.T = a->T; p.H = a->H; p.G = a->G; p.d = a->d; p.dv = a->dv; p.taps = a->taps; p.rot = a->rot; p.eps = a->eps;
  SX_ACT_DISPATCH(a->f32, {
    if (a->chunks.n == 0) return launch_qkv<A, 1, 8>(p, a->ragged.n, st);     // one row per portion
    if (!a->kv_row) return -3;
    return a->taps <= 4 ? launch_qkv<A, RC, 4>(p, a->chunks.n, st) : launch_qkv<A, RC, 8>(p, a->chunks.n, st);
  });
  return 0;
}
extern "C" int sx_kv_gather(const void* cache, const int* entry, const int* row, int n, void* out, long long out_ld, int G, int w,
                            int wp, int f32, cudaStream_t st) {
  if (n <= 0) return 0;
  SX_ACT_DISPATCH(f32, (kv_gather_kernel<A><<<n, 128, 0, st>>>((const A*)cache, entry, row, (A*)out, out_ld, G, w, wp)));
  return last_rc();
}
