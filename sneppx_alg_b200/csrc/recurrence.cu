// Gated linear recurrences with an fp32 state per head, S [d, dv]:
//   gated write   S <- f S + (1 - f) v^T                               o = S^T q        (decay f per row)
//   gated delta   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;     o = S^T q        (decay g per row)
// Operand preparation, the scan over a portion of a prompt, and the one-token step of decoding. The state stays in fp32
// and every term that enters it is computed in fp32; a portion may start from any stored state, so a prompt can be cut
// anywhere. State layout: [slots, H, d, dv].
#include "common.cuh"
#include "ragged.cuh"
#include "sx_api.h"

namespace sx {

// ------------------------------------------------------------------ gated delta rule operands
struct DeltaParams {
  const void* u;              // projected rows: q [G d] | k [G d] | v [H dv]
  long long u_ld;
  const float* wconv;         // [taps, C], C = 2 G d + H dv
  void* ring;                 // [slots, taps, C]
  const void* b; long long b_ld;      // [T, H] write-strength logits
  const void* a; long long a_ld;      // [T, H d] decay inputs (second low-rank product)
  const float* a_log; const float* dt_bias;   // [H], [H d]
  float* q; float* k;         // [T, G, d]
  float* g;                   // [T, H, d] decay
  void* v;                    // [T, H dv] activation type
  float* beta;                // [T, H]
  RaggedView rv;
  int T, H, G, d, dv, taps, write_ring;
};

template <typename A>
__device__ __forceinline__ float conv_silu_at(const DeltaParams& p, const A* __restrict__ row, int ch, int C, int pos, int pos0,
                                              const A* __restrict__ ring) {
  float acc = 0.f;
  for (int j = 0; j < p.taps; ++j) {
    const int b = p.taps - 1 - j;
    if (b > pos) continue;
    const float x = pos - b >= pos0 ? to_f(row[ch - (long long)b * p.u_ld]) : to_f(ring[(long long)((pos - b) % p.taps) * C + ch]);
    acc = fmaf(p.wconv[(long long)j * C + ch], x, acc);
  }
  return acc * sigmoid_f(acc);
}

template <typename A>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaParams p) {
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int seq = p.rv.tok_seq[t], pos = p.rv.tok_pos[t], pos0 = p.rv.pos0[seq];
  const int C = 2 * p.G * p.d + p.H * p.dv;
  const A* row = reinterpret_cast<const A*>(p.u) + (long long)t * p.u_ld;
  A* ring = reinterpret_cast<A*>(p.ring) + (long long)p.rv.slot[seq] * p.taps * C;
  for (int hh = warp; hh < 2 * p.G; hh += nw) {
    float v[2 * QK_PAIRS];
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < 2 * QK_PAIRS; ++n) {
      const int i = lane + 32 * n;
      v[n] = i < p.d ? conv_silu_at<A>(p, row, hh * p.d + i, C, pos, pos0, ring) : 0.f;
      ss += v[n] * v[n];
    }
    ss = warp_sum(ss);
    float r = 1.f / sqrtf(ss + 1e-6f);
    if (hh < p.G) r *= 1.f / sqrtf((float)p.d);
    float* out = (hh < p.G ? p.q + ((long long)t * p.G + hh) * p.d : p.k + ((long long)t * p.G + hh - p.G) * p.d);
#pragma unroll
    for (int n = 0; n < 2 * QK_PAIRS; ++n) {
      const int i = lane + 32 * n;
      if (i < p.d) out[i] = v[n] * r;
    }
  }
  for (int c = threadIdx.x; c < p.H * p.dv; c += blockDim.x)
    reinterpret_cast<A*>(p.v)[(long long)t * p.H * p.dv + c] =
        from_f<A>(conv_silu_at<A>(p, row, 2 * p.G * p.d + c, C, pos, pos0, ring));
  const A* ar = reinterpret_cast<const A*>(p.a) + (long long)t * p.a_ld;
  for (int c = threadIdx.x; c < p.H * p.d; c += blockDim.x) {
    const float z = to_f(ar[c]) + p.dt_bias[c];
    p.g[(long long)t * p.H * p.d + c] = expf(-expf(p.a_log[c / p.d]) * softplus_f(z));
  }
  for (int h = threadIdx.x; h < p.H; h += blockDim.x)
    p.beta[(long long)t * p.H + h] = sigmoid_f(to_f(reinterpret_cast<const A*>(p.b)[(long long)t * p.b_ld + h]));
  if (p.write_ring && p.taps > 1 && p.rv.slot[seq] >= 0)
    for (int c = threadIdx.x; c < C; c += blockDim.x) ring[(long long)(pos % p.taps) * C + c] = row[c];
}

// ------------------------------------------------------------------ gated-write recurrence operands
// q = silu(q_raw), f = lower + (1 - lower) sigmoid(f_raw + bias)
template <typename A>
__global__ void __launch_bounds__(256) gate_prep_kernel(const A* __restrict__ qr, const A* __restrict__ fr, long long ld,
                                                        const float* __restrict__ bias, const float* __restrict__ lower,
                                                        float* __restrict__ q, float* __restrict__ f, long long n, int C) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const long long t = i / C;
  const int c = (int)(i % C);
  const float z = to_f(qr[t * ld + c]);
  q[i] = z * sigmoid_f(z);
  const float l = lower[c];
  f[i] = l + (1.f - l) * sigmoid_f(to_f(fr[t * ld + c]) + bias[c]);
}

// ------------------------------------------------------------------ scan over the tokens of a portion
struct ScanParams {
  const float* q; const float* g; const float* k;   // [T, Hq, d], [T, H, d] decay, [T, Hq, d] (delta rule only)
  const void* v; long long v_ld;                    // [T, H dv]
  const float* beta;                                // [T, H] (delta rule only)
  float* state;                                     // [slots, H, d, dv]
  float* o;                                         // [T, H, dv]
  RaggedView rv;
  int H, Hq, d, dv;
};

typedef unsigned long long u64;
__device__ __forceinline__ u64 pack2(float lo, float hi) {
  u64 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unpack2(u64 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ u64 fma2(u64 a, u64 b, u64 c) {
  u64 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ u64 mul2(u64 a, u64 b) {
  u64 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// One CTA walks the tokens of one portion for one head and a tile of value columns. The state tile lives in registers:
// a thread holds 16 rows of CN columns, LANES neighbouring lanes share a column. Operand rows of TT tokens at a time are
// copied to shared memory ahead of their use. The read-out sums of LANES tokens are reduced across the lanes together
// (lane i ends up with token i), so they cost LANES - 1 shuffles per LANES tokens and stay off the recurrence's chain.
template <typename A, bool DELTA, int LANES, int CN>
struct ScanCfg {
  static constexpr int DP = LANES * 16;              // padded rows
  static constexpr int TT = DP <= 128 ? 16 : 8;
  static constexpr int CT = 4 * (32 / LANES) * CN;   // columns per CTA
  static constexpr int NARR = DELTA ? 3 : 2;
  static constexpr int BUF = NARR * TT * DP;         // floats per buffer
  static constexpr int VN = (TT * CT + 127) / 128;
  static constexpr int SMEM = (2 * BUF + 2 * TT * CT + 2 * TT) * 4;
};

template <typename A, bool DELTA, int LANES, int CN>
__global__ void __launch_bounds__(128) recur_scan_kernel(const ScanParams p) {
  using Cfg = ScanCfg<A, DELTA, LANES, CN>;
  constexpr int DP = Cfg::DP, TT = Cfg::TT, CT = Cfg::CT, BUF = Cfg::BUF, VN = Cfg::VN, GW = 32 / LANES;
  constexpr int STEP = LANES < TT ? LANES : TT;      // tokens whose read-outs are reduced together
  extern __shared__ __align__(16) float sm[];
  float* sOp = sm;                       // [2][NARR][TT][DP]: q, decay, k
  float* sV = sm + 2 * BUF;              // [2][TT][CT]
  float* sB = sV + 2 * TT * CT;          // [2][TT]
  const int seq = blockIdx.z, h = blockIdx.y, hq = h / (p.H / p.Hq);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rl = lane % LANES, cloc = (warp * GW + lane / LANES) * CN, c0 = blockIdx.x * CT;
  const int row0 = p.rv.cu[seq], len = p.rv.cu[seq + 1] - row0;
  if (len <= 0) return;
  float* st = p.state + ((long long)p.rv.slot[seq] * p.H + h) * p.d * p.dv;
  const bool fresh = p.rv.pos0[seq] == 0;

  u64 S[CN][8];
#pragma unroll
  for (int cn = 0; cn < CN; ++cn) {
    const int col = c0 + cloc + cn;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int r = (i / 2) * LANES * 4 + rl * 4 + (i % 2) * 2;
      float a = 0.f, b = 0.f;
      if (!fresh && col < p.dv) {
        if (r < p.d) a = st[(long long)r * p.dv + col];
        if (r + 1 < p.d) b = st[(long long)(r + 1) * p.dv + col];
      }
      S[cn][i] = pack2(a, b);
    }
  }
  if (p.d < DP)   // padding rows: zero operands, never overwritten
    for (int i = tid; i < 2 * Cfg::NARR * TT * (DP - p.d); i += 128) sOp[(i / (DP - p.d)) * DP + p.d + i % (DP - p.d)] = 0.f;

  const bool vec = (p.d & 3) == 0;
  auto fetch = [&](int t0, int buf) {
    const int nt = min(TT, len - t0);
    float* dst = sOp + buf * BUF;
#pragma unroll
    for (int a = 0; a < Cfg::NARR; ++a) {
      const float* src = a == 0 ? p.q : (a == 1 ? p.g : p.k);
      const int heads = a == 1 ? p.H : p.Hq, hh = a == 1 ? h : hq;
      if (vec) {
        const int per = p.d / 4;
        for (int i = tid; i < nt * per; i += 128) {
          const int t = i / per, c = (i % per) * 4;
          cp_async16(dst + (a * TT + t) * DP + c, src + ((long long)(row0 + t0 + t) * heads + hh) * p.d + c);
        }
      } else {
        for (int i = tid; i < nt * p.d; i += 128) {
          const int t = i / p.d, c = i % p.d;
          cp_async4(dst + (a * TT + t) * DP + c, src + ((long long)(row0 + t0 + t) * heads + hh) * p.d + c);
        }
      }
    }
    cp_async_commit();
  };
  float vreg[VN], breg = 0.f;
  auto load_v = [&](int t0) {
    const int nt = min(TT, len - t0);
#pragma unroll
    for (int n = 0; n < VN; ++n) {
      const int i = tid + n * 128, t = i / CT, c = c0 + i % CT;
      vreg[n] = (i < TT * CT && t < nt && c < p.dv)
                    ? to_f(reinterpret_cast<const A*>(p.v)[(long long)(row0 + t0 + t) * p.v_ld + (long long)h * p.dv + c])
                    : 0.f;
    }
    if (DELTA && tid < TT) breg = tid < nt ? p.beta[(long long)(row0 + t0 + tid) * p.H + h] : 0.f;
  };
  auto put_v = [&](int buf) {
#pragma unroll
    for (int n = 0; n < VN; ++n) {
      const int i = tid + n * 128;
      if (i < TT * CT) sV[buf * TT * CT + i] = vreg[n];
    }
    if (DELTA && tid < TT) sB[buf * TT + tid] = breg;
  };

  const u64 one2 = pack2(1.f, 1.f), neg2 = pack2(-1.f, -1.f);
  fetch(0, 0);
  load_v(0);
  put_v(0);
  int buf = 0;
  for (int t0 = 0; t0 < len; t0 += TT, buf ^= 1) {
    const int nt = min(TT, len - t0);
    const bool more = t0 + TT < len;
    if (more) {
      fetch(t0 + TT, buf ^ 1);
      load_v(t0 + TT);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* op = sOp + buf * BUF + rl * 4;
    const float* vp = sV + buf * TT * CT + cloc;
    for (int ts = 0; ts < nt; ts += STEP) {
      float oacc[CN][STEP];
#pragma unroll
      for (int s = 0; s < STEP; ++s) {
        const int t = ts + s;
#pragma unroll
        for (int cn = 0; cn < CN; ++cn) oacc[cn][s] = 0.f;
        if (t < nt) {
          u64 q[8], g[8], k[8];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(op + t * DP + c * LANES * 4);
            const ulonglong2 g4 = *reinterpret_cast<const ulonglong2*>(op + (TT + t) * DP + c * LANES * 4);
            q[2 * c] = q4.x; q[2 * c + 1] = q4.y;
            g[2 * c] = g4.x; g[2 * c + 1] = g4.y;
            if constexpr (DELTA) {
              const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(op + (2 * TT + t) * DP + c * LANES * 4);
              k[2 * c] = k4.x; k[2 * c + 1] = k4.y;
            } else {
              k[2 * c] = fma2(g4.x, neg2, one2);
              k[2 * c + 1] = fma2(g4.y, neg2, one2);
            }
          }
          if constexpr (DELTA) {
            const float beta = sB[buf * TT + t];
            float w[CN];
#pragma unroll
            for (int cn = 0; cn < CN; ++cn) {
              u64 a0 = 0, a1 = 0;
#pragma unroll
              for (int i = 0; i < 8; i += 2) {
                S[cn][i] = mul2(g[i], S[cn][i]);
                S[cn][i + 1] = mul2(g[i + 1], S[cn][i + 1]);
                a0 = fma2(S[cn][i], k[i], a0);
                a1 = fma2(S[cn][i + 1], k[i + 1], a1);
              }
              const float2 x = unpack2(a0), y = unpack2(a1);
              w[cn] = (x.x + x.y) + (y.x + y.y);
            }
#pragma unroll
            for (int m = LANES / 2; m >= 1; m >>= 1)
#pragma unroll
              for (int cn = 0; cn < CN; ++cn) w[cn] += __shfl_xor_sync(0xffffffffu, w[cn], m);
#pragma unroll
            for (int cn = 0; cn < CN; ++cn) {
              const float u = beta * (vp[t * CT + cn] - w[cn]);
              const u64 u2 = pack2(u, u);
              u64 a0 = 0, a1 = 0;
#pragma unroll
              for (int i = 0; i < 8; i += 2) {
                S[cn][i] = fma2(k[i], u2, S[cn][i]);
                S[cn][i + 1] = fma2(k[i + 1], u2, S[cn][i + 1]);
                a0 = fma2(S[cn][i], q[i], a0);
                a1 = fma2(S[cn][i + 1], q[i + 1], a1);
              }
              const float2 x = unpack2(a0), y = unpack2(a1);
              oacc[cn][s] = (x.x + x.y) + (y.x + y.y);
            }
          } else {
#pragma unroll
            for (int cn = 0; cn < CN; ++cn) {
              const float v = vp[t * CT + cn];
              const u64 v2 = pack2(v, v);
              u64 a0 = 0, a1 = 0;
#pragma unroll
              for (int i = 0; i < 8; i += 2) {
                S[cn][i] = fma2(g[i], S[cn][i], mul2(k[i], v2));
                S[cn][i + 1] = fma2(g[i + 1], S[cn][i + 1], mul2(k[i + 1], v2));
                a0 = fma2(S[cn][i], q[i], a0);
                a1 = fma2(S[cn][i + 1], q[i + 1], a1);
              }
              const float2 x = unpack2(a0), y = unpack2(a1);
              oacc[cn][s] = (x.x + x.y) + (y.x + y.y);
            }
          }
        }
      }
      // token-transposed reduction over the lanes that share a column (LANES can exceed STEP: plain steps first)
#pragma unroll
      for (int cn = 0; cn < CN; ++cn) {
#pragma unroll
        for (int m = LANES / 2; m >= STEP && m >= 1; m >>= 1)
#pragma unroll
          for (int s = 0; s < STEP; ++s) oacc[cn][s] += __shfl_xor_sync(0xffffffffu, oacc[cn][s], m);
#pragma unroll
        for (int m = STEP / 2; m >= 1; m >>= 1) {
          const bool up = (rl & m) != 0;
#pragma unroll
          for (int s = 0; s < m; ++s) {
            const float mine = up ? oacc[cn][s + m] : oacc[cn][s], other = up ? oacc[cn][s] : oacc[cn][s + m];
            oacc[cn][s] = mine + __shfl_xor_sync(0xffffffffu, other, m);
          }
        }
        const int t = ts + rl % STEP, col = c0 + cloc + cn;
        if (rl < STEP && t < nt && col < p.dv) p.o[((long long)(row0 + t0 + t) * p.H + h) * p.dv + col] = oacc[cn][0];
      }
    }
    if (more) put_v(buf ^ 1);
    __syncthreads();
  }
#pragma unroll
  for (int cn = 0; cn < CN; ++cn) {
    const int col = c0 + cloc + cn;
    if (col >= p.dv) continue;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int r = (i / 2) * LANES * 4 + rl * 4 + (i % 2) * 2;
      const float2 x = unpack2(S[cn][i]);
      if (r < p.d) st[(long long)r * p.dv + col] = x.x;
      if (r + 1 < p.d) st[(long long)(r + 1) * p.dv + col] = x.y;
    }
  }
}

// ------------------------------------------------------------------ one token per sequence
// One CTA per (head, sequence): operands from the projected rows (convolution, unit norms, gates), one state update with
// the state tile in registers between its two passes, read-out, per-head norm and output gate.
struct StepParams {
  DeltaParams in;             // delta rule: projected rows and constants (q, k, g, v, beta unused)
  const void* qr; const void* fr; const void* vr; long long ld;   // gated write: projected rows
  const float* fbias; const float* lower;
  float* state;
  const float* norm;          // [dv]
  const void* gate; long long gate_ld;   // null: no output gate
  void* y; long long y_ld;
  float mul, eps;
  RaggedView rv;
  int H, Hq, d, dv, lpr;      // lpr: lanes that share a state row
};

template <typename A, bool DELTA, int VEC, int NR>
__global__ void __launch_bounds__(256) recur_step_kernel(const StepParams p) {
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;             // [d]
  float* sk = sq + p.d;       // [d]
  float* sg = sk + p.d;       // [d]
  float* sv = sg + p.d;       // [dv]
  float* so = sv + p.dv;      // [dv]
  float* red = so + p.dv;     // [8][32 * VEC] partial sums, or 40 scratch floats
  const int h = blockIdx.x, seq = blockIdx.y, hq = h / (p.H / p.Hq);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t = p.rv.cu[seq];
  const int slot = p.rv.slot[seq];
  if (slot < 0) return;       // padding row of a captured launch
  const int pos = p.rv.pos0[seq];
  float beta = 0.f;
  if constexpr (DELTA) {
    const DeltaParams& in = p.in;
    const int C = 2 * in.G * in.d + in.H * in.dv;
    const A* row = reinterpret_cast<const A*>(in.u) + (long long)t * in.u_ld;
    A* ring = reinterpret_cast<A*>(in.ring) + (long long)slot * in.taps * C;
    if (warp < 2) {           // warp 0: query, warp 1: key
      const int ch0 = (warp * in.G + hq) * in.d;
      float ss = 0.f;
      float* dst = warp ? sk : sq;
      for (int i = lane; i < in.d; i += 32) {
        const float x = conv_silu_at<A>(in, row, ch0 + i, C, pos, pos, ring);
        dst[i] = x;
        ss += x * x;
      }
      ss = warp_sum(ss);
      float r = 1.f / sqrtf(ss + 1e-6f);
      if (warp == 0) r *= 1.f / sqrtf((float)in.d);
      for (int i = lane; i < in.d; i += 32) dst[i] *= r;
    } else if (warp < 5) {
      for (int c = tid - 64; c < in.dv; c += 96)
        sv[c] = to_f(from_f<A>(conv_silu_at<A>(in, row, 2 * in.G * in.d + h * in.dv + c, C, pos, pos, ring)));
    } else {
      const A* ar = reinterpret_cast<const A*>(in.a) + (long long)t * in.a_ld + (long long)h * in.d;
      const float al = -expf(in.a_log[h]);
      for (int i = tid - 160; i < in.d; i += 96) sg[i] = expf(al * softplus_f(to_f(ar[i]) + in.dt_bias[h * in.d + i]));
    }
    beta = sigmoid_f(to_f(reinterpret_cast<const A*>(in.b)[(long long)t * in.b_ld + h]));
    if (in.taps > 1) {
      // the entry this token fills is not one that any head reads in this step
      A* e = ring + (long long)(pos % in.taps) * C;
      if (h % (p.H / p.Hq) == 0)
        for (int i = tid; i < 2 * in.d; i += 256) {
          const int ch = ((i / in.d) * in.G + hq) * in.d + i % in.d;
          e[ch] = row[ch];
        }
      for (int c = tid; c < in.dv; c += 256) {
        const int ch = 2 * in.G * in.d + h * in.dv + c;
        e[ch] = row[ch];
      }
    }
  } else {
    const A* qr = reinterpret_cast<const A*>(p.qr) + (long long)t * p.ld + (long long)h * p.d;
    const A* fr = reinterpret_cast<const A*>(p.fr) + (long long)t * p.ld + (long long)h * p.d;
    const A* vr = reinterpret_cast<const A*>(p.vr) + (long long)t * p.ld + (long long)h * p.dv;
    for (int i = tid; i < p.d; i += 256) {
      const float z = to_f(qr[i]);
      sq[i] = z * sigmoid_f(z);
      const float l = p.lower[h * p.d + i];
      const float f = l + (1.f - l) * sigmoid_f(to_f(fr[i]) + p.fbias[h * p.d + i]);
      sg[i] = f;
      sk[i] = 1.f - f;
    }
    for (int c = tid; c < p.dv; c += 256) sv[c] = to_f(vr[c]);
  }
  __syncthreads();

  const int lpr = p.lpr, RG = 256 / lpr, rg = tid / lpr, cl = tid % lpr;
  float* st = p.state + ((long long)slot * p.H + h) * p.d * p.dv;
  const bool fresh = pos == 0;
  for (int ct = 0; ct < p.dv; ct += lpr * VEC) {
    const int col = ct + cl * VEC;
    const bool on = col < p.dv;
    float S[NR][VEC];
#pragma unroll
    for (int n = 0; n < NR; ++n) {
      const int r = rg + n * RG;
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[n][e] = 0.f;
      if (!fresh && on && r < p.d) {
        if constexpr (VEC == 4) {
          const float4 x = *reinterpret_cast<const float4*>(st + (long long)r * p.dv + col);
          S[n][0] = x.x; S[n][1] = x.y; S[n][2] = x.z; S[n][3] = x.w;
        } else {
          S[n][0] = st[(long long)r * p.dv + col];
        }
      }
    }
    // sum over the state rows of acc[VEC], result for this thread's columns in every thread
    auto reduce = [&](float (&acc)[VEC]) {
      for (int m = lpr; m < 32; m <<= 1)
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], m);
      __syncthreads();
      if (lane < lpr)
#pragma unroll
        for (int e = 0; e < VEC; ++e) red[warp * 32 * VEC + cl * VEC + e] = acc[e];
      __syncthreads();
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) s += red[w * 32 * VEC + cl * VEC + e];
        acc[e] = s;
      }
    };
    float u[VEC], acc[VEC];
    if constexpr (DELTA) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
#pragma unroll
      for (int n = 0; n < NR; ++n) {
        const int r = rg + n * RG;
        if (r < p.d) {
          const float g = sg[r], k = sk[r];
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            S[n][e] *= g;
            acc[e] = fmaf(S[n][e], k, acc[e]);
          }
        }
      }
      reduce(acc);
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[e] = on ? beta * (sv[col + e] - acc[e]) : 0.f;
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[e] = on ? sv[col + e] : 0.f;
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
#pragma unroll
    for (int n = 0; n < NR; ++n) {
      const int r = rg + n * RG;
      if (r < p.d) {
        const float k = sk[r], q = sq[r], g = DELTA ? 1.f : sg[r];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          S[n][e] = DELTA ? fmaf(k, u[e], S[n][e]) : fmaf(g, S[n][e], k * u[e]);
          acc[e] = fmaf(S[n][e], q, acc[e]);
        }
        if (on) {
          if constexpr (VEC == 4) *reinterpret_cast<float4*>(st + (long long)r * p.dv + col) = make_float4(S[n][0], S[n][1], S[n][2], S[n][3]);
          else st[(long long)r * p.dv + col] = S[n][0];
        }
      }
    }
    reduce(acc);
    if (rg == 0 && on)
#pragma unroll
      for (int e = 0; e < VEC; ++e) so[col + e] = acc[e];
    __syncthreads();
  }
  float ss = 0.f;
  for (int c = tid; c < p.dv; c += 256) ss += so[c] * so[c];
  ss = block_sum(ss, red);
  const float r = p.mul / sqrtf(ss / p.dv + p.eps);
  A* y = reinterpret_cast<A*>(p.y) + (long long)t * p.y_ld + (long long)h * p.dv;
  const A* gr = p.gate ? reinterpret_cast<const A*>(p.gate) + (long long)t * p.gate_ld + (long long)h * p.dv : nullptr;
  for (int c = tid; c < p.dv; c += 256) {
    float v = so[c] * r * p.norm[c];
    if (gr) v *= sigmoid_f(to_f(gr[c]));
    y[c] = from_f<A>(v);
  }
}

}  // namespace sx
using namespace sx;

static void fill_delta(DeltaParams* p, const SxDeltaArgs* a) {
  p->u = a->u; p->u_ld = a->u_ld; p->wconv = a->wconv; p->ring = a->ring; p->b = a->b; p->b_ld = a->b_ld; p->a = a->a; p->a_ld = a->a_ld;
  p->a_log = a->a_log; p->dt_bias = a->dt_bias; p->q = a->q; p->k = a->k; p->g = a->g; p->v = a->v; p->beta = a->beta;
  p->rv = view(&a->ragged);
  p->T = a->T; p->H = a->H; p->G = a->G; p->d = a->d; p->dv = a->dv; p->taps = a->taps; p->write_ring = a->write_ring;
}
extern "C" int sx_delta_prep(const SxDeltaArgs* a, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (a->d > 64 * QK_PAIRS || a->G <= 0 || a->H % a->G) return -1;
  DeltaParams p;
  fill_delta(&p, a);
  SX_ACT_DISPATCH(a->f32, (delta_prep_kernel<A><<<a->T, 256, 0, st>>>(p)));
  return last_rc();
}
extern "C" int sx_gate_prep(const void* qr, const void* fr, long long ld, const float* bias, const float* lower, float* q, float* f,
                            int T, int C, int f32, cudaStream_t st) {
  const long long n = (long long)T * C;
  if (n <= 0) return 0;
  SX_ACT_DISPATCH(f32, (gate_prep_kernel<A><<<(unsigned)((n + 255) / 256), 256, 0, st>>>((const A*)qr, (const A*)fr, ld, bias, lower, q, f, n, C)));
  return last_rc();
}

template <typename A, bool DELTA, int LANES, int CN>
static int launch_scan(const ScanParams& p, cudaStream_t st) {
  using Cfg = ScanCfg<A, DELTA, LANES, CN>;
  static bool set = false;
  if (!set) {
    if (cudaFuncSetAttribute(recur_scan_kernel<A, DELTA, LANES, CN>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM) != cudaSuccess)
      return -10;
    set = true;
  }
  dim3 grid((p.dv + Cfg::CT - 1) / Cfg::CT, p.H, p.rv.n);
  recur_scan_kernel<A, DELTA, LANES, CN><<<grid, 128, Cfg::SMEM, st>>>(p);
  return last_rc();
}
template <typename A, bool DELTA>
static int pick_scan(const ScanParams& p, cudaStream_t st) {
  // two columns per thread once one column per thread would put more than two CTAs on every SM
  const int lanes = p.d <= 16 ? 1 : p.d <= 32 ? 2 : p.d <= 64 ? 4 : p.d <= 128 ? 8 : 16;
  const int ct1 = 4 * (32 / lanes);
  const bool wide = (long long)((p.dv + ct1 - 1) / ct1) * p.H * p.rv.n > 2 * 148;
#define SX_SCAN(L) return wide ? launch_scan<A, DELTA, L, 2>(p, st) : launch_scan<A, DELTA, L, 1>(p, st)
  switch (lanes) {
    case 1: SX_SCAN(1);
    case 2: SX_SCAN(2);
    case 4: SX_SCAN(4);
    case 8: SX_SCAN(8);
    default: SX_SCAN(16);
  }
#undef SX_SCAN
}

// delta != 0: gated delta rule; else the gated write. The portion's rows must be in order; portions are independent.
extern "C" int sx_recur_scan(const SxScanArgs* a, cudaStream_t st) {
  if (a->ragged.n <= 0) return 0;
  if (a->d <= 0 || a->d > 256 || a->dv <= 0 || a->Hq <= 0 || a->H % a->Hq) return -1;
  ScanParams p;
  p.q = a->q; p.g = a->g; p.k = a->k; p.v = a->v; p.v_ld = a->v_ld; p.beta = a->beta; p.state = a->state; p.o = a->o;
  p.rv = view(&a->ragged);
  p.H = a->H; p.Hq = a->Hq; p.d = a->d; p.dv = a->dv;
  SX_ACT_DISPATCH(a->f32, { return a->delta ? pick_scan<A, true>(p, st) : pick_scan<A, false>(p, st); });
  return 0;
}

template <typename A, bool DELTA, int VEC>
static int launch_step(const StepParams& p, cudaStream_t st) {
  const int rows = 256 / p.lpr, nr = (p.d + rows - 1) / rows;
  const int smem = (3 * p.d + 2 * p.dv + 8 * 32 * VEC + 40) * 4;
  if (smem > 48 * 1024) return -2;
  const dim3 grid(p.H, p.rv.n);
  if (nr <= 4) recur_step_kernel<A, DELTA, VEC, 4><<<grid, 256, smem, st>>>(p);
  else if (nr <= 8) recur_step_kernel<A, DELTA, VEC, 8><<<grid, 256, smem, st>>>(p);
  else if (nr <= 16) recur_step_kernel<A, DELTA, VEC, 16><<<grid, 256, smem, st>>>(p);
  else if (nr <= 32) recur_step_kernel<A, DELTA, VEC, 32><<<grid, 256, smem, st>>>(p);
  else return -3;
  return last_rc();
}

extern "C" int sx_recur_step(const SxStepArgs* a, cudaStream_t st) {
  if (a->ragged.n <= 0) return 0;
  if (a->d <= 0 || a->d > 256 || a->dv <= 0 || a->Hq <= 0 || a->H % a->Hq) return -1;
  StepParams p;
  p.rv = view(&a->ragged);
  if (a->delta) {
    const SxDeltaArgs* d = &a->in;
    fill_delta(&p.in, d);
  }
  p.qr = a->qr; p.fr = a->fr; p.vr = a->vr; p.ld = a->ld; p.fbias = a->fbias; p.lower = a->lower;
  p.state = a->state; p.norm = a->norm; p.gate = a->gate; p.gate_ld = a->gate_ld; p.y = a->y; p.y_ld = a->y_ld;
  p.mul = a->mul; p.eps = a->eps; p.H = a->H; p.Hq = a->Hq; p.d = a->d; p.dv = a->dv;
  const int vec = (a->dv % 4 == 0) ? 4 : 1, cv = (a->dv + vec - 1) / vec;
  p.lpr = cv >= 32 ? 32 : cv > 16 ? 32 : cv > 8 ? 16 : cv > 4 ? 8 : 4;
  SX_ACT_DISPATCH(a->f32, {
    if (a->delta) return vec == 4 ? launch_step<A, true, 4>(p, st) : launch_step<A, true, 1>(p, st);
    return vec == 4 ? launch_step<A, false, 4>(p, st) : launch_step<A, false, 1>(p, st);
  });
  return 0;
}
