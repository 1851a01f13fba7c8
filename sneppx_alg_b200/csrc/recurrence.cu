// Gated linear recurrences with an fp32 state per head, S [d, dv]:
//   gated write   S <- f S + (1 - f) v^T                               o = S^T q        (decay f per row)
//   SSD           S <- a S + dt B x^T                                  o = S^T C        (one decay a per head; prompts of
//                                                                       32-bit runs, the other forms are in ssd_serve.cu)
//   gated delta   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;     o = S^T q        (decay g per row)
// Operand preparation, the scan over a portion of a prompt, and the one-token step of decoding. The state stays in fp32
// and every term that enters it is computed in fp32; a portion may start from any stored state, so a prompt can be cut
// anywhere. State layout: [slots, H, d, dv].
#include "common.cuh"
#include "ragged.cuh"
#include "tc_common.cuh"
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
  void* v;                    // [T, H dv] convolved values, activation type
  RaggedView rv;
  int T, H, G, d, dv, taps;
};

// ------------------------------------------------------------------ chunk form of the recurrences
// A portion is walked in chunks of RC tokens. With G_t the product of the decays of the chunk's tokens up to t, the state
// S0 in front of the chunk and k_t, u_t the written key and value,
//   o_t = S0^T (G_t q_t) + sum_{i <= t} B_ti u_i,          B_ti = q_t . (prod_{i < j <= t} g_j) k_i
//   S   = G_last S0 + sum_t (prod_{j > t} g_j) k_t u_t^T
// u_t is v_t for the gated write; for the delta rule (I + diag(beta) A) U = diag(beta) (V - S0^T (G k)) with A_ti the
// strictly lower part of k_t . (prod g) k_i, and the inverse is formed once per chunk and head. Products of decays are
// formed by multiplication only, so no decay is ever divided out. A preparation kernel writes everything of a (chunk,
// head) that does not depend on the state as one contiguous record of fp32 values:
//   Gq [RC, DP] | Kd [RC, DP] | Gk [RC, DP] (delta) | G_last [DP] | B [RC, RC] | (I + diag(beta) A)^-1 diag(beta) (delta)
// with padded row pitches (DP + 8, DP + 4, DP + 8; RC + 8) that keep the tensor-core kernel's fragment reads free of bank
// conflicts.
template <int DP, bool DELTA>
struct Rec {
  static constexpr int LQ = DP + 8, LK = DP + 4, LB = RC + 8;
  static constexpr int KD = RC * LQ, GK = KD + RC * LK, GL = GK + (DELTA ? RC * LQ : 0), B = GL + DP, TM = B + RC * LB;
  static constexpr int FLOATS = TM + (DELTA ? RC * LB : 0);
};

// Sums of v[16] over the lanes that share a column group (LANES neighbouring lanes): lane rl is left with the sums of
// tokens rl * TPL .. rl * TPL + TPL - 1 in v[0 .. TPL).
template <int LANES>
__device__ __forceinline__ void reduce_tokens(float (&v)[RC], int rl) {
  int n = RC;
#pragma unroll
  for (int m = LANES / 2; m >= 1; m >>= 1) {
    n >>= 1;
    const bool up = (rl & m) != 0;
#pragma unroll
    for (int i = 0; i < RC / 2; ++i)
      if (i < n) {
        const float mine = up ? v[i + n] : v[i], other = up ? v[i] : v[i + n];
        v[i] = mine + __shfl_xor_sync(0xffffffffu, other, m);
      }
  }
}

// Writes the record from q, k, g [RC][DP] in shared memory (rows past nt and columns past d: q = k = 0, g = 1 resp. 0).
template <int DP, bool DELTA>
__device__ __forceinline__ void write_record(const float* __restrict__ sq, const float* __restrict__ sk, const float* __restrict__ sg,
                                             const float* __restrict__ sbeta, float* __restrict__ sA, float* __restrict__ rec, int nt) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  using R = Rec<DP, DELTA>;
  float* Gq = rec;
  float* Kd = rec + R::KD;
  float* Gk = rec + R::GK;
  float* Gl = rec + R::GL;
  float* B = rec + R::B;
  float* Tm = rec + R::TM;
  for (int i = tid; i < 2 * DP; i += 256) {
    const int c = i % DP;
    float p = 1.f;
    if (i < DP) {
#pragma unroll
      for (int t = 0; t < RC; ++t) {
        p *= sg[t * DP + c];
        Gq[t * R::LQ + c] = sq[t * DP + c] * p;
        if (DELTA) Gk[t * R::LQ + c] = sk[t * DP + c] * p;
      }
      Gl[c] = p;
    } else {
#pragma unroll
      for (int t = RC - 1; t >= 0; --t) {
        Kd[t * R::LK + c] = sk[t * DP + c] * p;
        p *= sg[t * DP + c];
      }
    }
  }
  constexpr int NC = (DP + 31) / 32;
#pragma unroll 1
  for (int half = 0; half < 2; ++half) {
    const int t = half ? RC - 1 - warp : warp;     // a warp takes a short and a long row
    float qp[NC], kp[NC], bq[RC], ak[RC];
#pragma unroll
    for (int n = 0; n < NC; ++n) {
      const int c = lane + 32 * n;
      qp[n] = c < DP ? sq[t * DP + c] : 0.f;
      if (DELTA) kp[n] = c < DP ? sk[t * DP + c] : 0.f;
    }
#pragma unroll
    for (int i = RC - 1; i >= 0; --i) {
      bq[i] = ak[i] = 0.f;
      if (i > t) continue;
#pragma unroll
      for (int n = 0; n < NC; ++n) {
        const int c = lane + 32 * n;
        {
          const float k = sk[i * DP + c], g = sg[i * DP + c];
          bq[i] = fmaf(qp[n], k, bq[i]);
          qp[n] *= g;
          if (DELTA) {
            ak[i] = fmaf(kp[n], k, ak[i]);
            kp[n] *= g;
          }
        }
      }
    }
    // over 32 lanes: the halves first, then the transposed reduction over 16 lanes
#pragma unroll
    for (int i = 0; i < RC; ++i) bq[i] += __shfl_xor_sync(0xffffffffu, bq[i], 16);
    reduce_tokens<16>(bq, lane & 15);
    if (lane < 16) B[t * R::LB + lane] = lane <= t ? bq[0] : 0.f;
    if constexpr (DELTA) {
#pragma unroll
      for (int i = 0; i < RC; ++i) ak[i] += __shfl_xor_sync(0xffffffffu, ak[i], 16);
      reduce_tokens<16>(ak, lane & 15);
      if (lane < 16) sA[t * RC + lane] = lane < t ? ak[0] : 0.f;
    }
  }
  if constexpr (DELTA) {
    __syncthreads();
    if (tid < RC) {        // column tid of the inverse, by forward substitution
      float x[RC];
#pragma unroll
      for (int t = 0; t < RC; ++t) {
        float s = t == tid ? 1.f : 0.f;
#pragma unroll
        for (int i = 0; i < t; ++i) s = fmaf(-sA[t * RC + i], x[i], s);
        x[t] = sbeta[t] * s;
        Tm[t * R::LB + tid] = x[t];
      }
    }
  }
}

template <typename A, int DP>
__global__ void __launch_bounds__(256) gate_chunk_kernel(const A* __restrict__ qr, const A* __restrict__ fr, long long ld,
                                                         const float* __restrict__ bias, const float* __restrict__ lower,
                                                         float* __restrict__ rec, const RaggedView rv, const ChunkView cv, int H, int d) {
  extern __shared__ __align__(128) float sm[];
  float* sq = sm;
  float* sk = sq + RC * DP;
  float* sg = sk + RC * DP;
  const int ch = blockIdx.x, h = blockIdx.y, seq = cv.seq[ch], s0 = cv.start[ch];
  const int row0 = rv.cu[seq] + s0, nt = min(RC, rv.cu[seq + 1] - row0);
#pragma unroll 4
  for (int i = threadIdx.x; i < RC * DP; i += 256) {
    const int t = i / DP, c = i % DP;
    float q = 0.f, f = 1.f;
    if (t < nt && c < d) {
      const long long o = (long long)(row0 + t) * ld + h * d + c;
      const float z = to_f(qr[o]), l = lower[h * d + c];
      q = silu_act<A>(z);
      f = l + (1.f - l) * sigmoid_f(to_f(fr[o]) + bias[h * d + c]);
    }
    sq[i] = q;
    sg[i] = f;
    sk[i] = 1.f - f;       // 0 on padding
  }
  __syncthreads();
  write_record<DP, false>(sq, sk, sg, nullptr, nullptr, rec + ((long long)ch * H + h) * Rec<DP, false>::FLOATS, nt);
}

// SSD records from the operands of sx_ssd_operands: q = C, k = dt B, one decay for all rows of a head's state.
template <typename A, int DP>
__global__ void __launch_bounds__(256) ssd_chunk_kernel(const A* __restrict__ b, const A* __restrict__ c, const float* __restrict__ dt,
                                                        const float* __restrict__ la, float* __restrict__ rec, const RaggedView rv,
                                                        const ChunkView cv, int H, int G, int N, int np) {
  extern __shared__ __align__(128) float sm[];
  float* sq = sm;
  float* sk = sq + RC * DP;
  float* sg = sk + RC * DP;
  const int ch = blockIdx.x, h = blockIdx.y, seq = cv.seq[ch], s0 = cv.start[ch];
  const int row0 = rv.cu[seq] + s0, nt = min(RC, rv.cu[seq + 1] - row0), g = h / (H / G);
  for (int i = threadIdx.x; i < RC * DP; i += 256) {
    const int t = i / DP, n = i % DP;
    float q = 0.f, k = 0.f, f = 1.f;
    if (t < nt) {
      const long long th = (long long)(row0 + t) * H + h;
      f = expf(la[th]);
      if (n < N) {
        const long long o = ((long long)(row0 + t) * G + g) * np + n;
        q = to_f(c[o]);
        k = to_f(b[o]) * dt[th];
      }
    }
    sq[i] = q;
    sk[i] = k;
    sg[i] = f;
  }
  __syncthreads();
  write_record<DP, false>(sq, sk, sg, nullptr, nullptr, rec + ((long long)ch * H + h) * Rec<DP, false>::FLOATS, nt);
}

template <typename A, int DP, int MT>
__global__ void __launch_bounds__(256, MT <= 4 && DP <= 128 ? 4 : 1) delta_chunk_kernel(const DeltaParams p, float* __restrict__ rec, const ChunkView cv) {
  extern __shared__ __align__(128) float sm[];
  float* sq = sm;
  float* sk = sq + RC * DP;
  float* sg = sk + RC * DP;
  float* sA = sg + RC * DP;            // [RC, RC]
  float* sb = sA + RC * RC;            // [RC]
  const int ch = blockIdx.x, h = blockIdx.y, hq = h / (p.H / p.G), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = cv.seq[ch], s0 = cv.start[ch], row0 = p.rv.cu[seq] + s0, nt = min(RC, p.rv.cu[seq + 1] - row0);
  const int pos = p.rv.pos0[seq] + s0, C = 2 * p.G * p.d + p.H * p.dv;
  const A* u = reinterpret_cast<const A*>(p.u) + (long long)row0 * p.u_ld;
  const A* ring = reinterpret_cast<const A*>(p.ring) + (long long)p.rv.slot[seq] * p.taps * C;
  // decay inputs and write strengths: in flight while the convolutions run
  constexpr int NA = RC * DP / 256;
  const A* ar = reinterpret_cast<const A*>(p.a) + (long long)row0 * p.a_ld + (long long)h * p.d;
  A av[NA], bv = from_f<A>(0.f);
#pragma unroll
  for (int n = 0; n < NA; ++n) {
    const int t = (tid + n * 256) / DP, c = tid % DP;
    av[n] = (t < nt && c < p.d) ? ar[(long long)t * p.a_ld + c] : from_f<A>(0.f);
  }
  if (tid < nt) bv = reinterpret_cast<const A*>(p.b)[(long long)(row0 + tid) * p.b_ld + h];
  for (int i = tid; i < 2 * DP + p.dv; i += 256) {
    const bool is_v = i >= 2 * DP;
    const int which = i / DP, c = is_v ? i - 2 * DP : i % DP;
    float y[RC];
    if (is_v || c < p.d) {
      const int col = is_v ? 2 * p.G * p.d + h * p.dv + c : (which * p.G + hq) * p.d + c;
      conv_walk<A, RC, MT>(u, p.u_ld, p.wconv, p.taps, C, col, ring, pos, s0, nt, y);
#pragma unroll
      for (int t = 0; t < RC; ++t) y[t] = silu_act<A>(y[t]);
    } else {
#pragma unroll
      for (int t = 0; t < RC; ++t) y[t] = 0.f;
    }
    if (is_v) {
      A* v = reinterpret_cast<A*>(p.v) + (long long)row0 * p.H * p.dv + (long long)h * p.dv + c;
#pragma unroll
      for (int t = 0; t < RC; ++t)
        if (t < nt) v[(long long)t * p.H * p.dv] = from_f<A>(y[t]);
    } else {
      float* dst = which ? sk : sq;
#pragma unroll
      for (int t = 0; t < RC; ++t) dst[t * DP + c] = t < nt ? y[t] : 0.f;
    }
  }
  const float al = -expf(p.a_log[h]);
#pragma unroll
  for (int n = 0; n < NA; ++n) {
    const int i = tid + n * 256, t = i / DP, c = i % DP;
    sg[i] = (t < nt && c < p.d) ? expf(al * softplus_f(to_f(av[n]) + p.dt_bias[h * p.d + c])) : 1.f;
  }
  if (tid < RC) sb[tid] = tid < nt ? sigmoid_f(to_f(bv)) : 0.f;
  __syncthreads();
  const float qs = 1.f / sqrtf((float)p.d);
  for (int i = warp; i < 2 * RC; i += 8) {
    float* row = (i < RC ? sq + i * DP : sk + (i - RC) * DP);
    float ss = 0.f;
    for (int c = lane; c < DP; c += 32) ss += row[c] * row[c];
    ss = warp_sum(ss);
    const float r = (i < RC ? qs : 1.f) / sqrtf(ss + 1e-6f);
    for (int c = lane; c < DP; c += 32) row[c] *= r;
  }
  __syncthreads();
  write_record<DP, true>(sq, sk, sg, sb, sA, rec + ((long long)ch * p.H + h) * Rec<DP, true>::FLOATS, nt);
}

// ------------------------------------------------------------------ scan over the chunks of a portion
struct ScanParams {
  const float* rec;
  const void* v; long long v_ld;                    // [T, H dv]
  float* state;                                     // [slots, H, d, dv]
  float* o;                                         // [T, H, dv]
  RaggedView rv;
  ChunkView cv;
  int* status;
  int H, d, dv;
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
__device__ __forceinline__ void bulk_load(void* dst, const void* src, unsigned bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

// One CTA walks one portion for one head and a tile of value columns. The state tile lives in registers: a thread holds 16
// rows of CN columns, LANES neighbouring lanes share a column. Records arrive by bulk copies one chunk ahead. A column
// belongs to one warp, so the exchange of written values inside a chunk needs no block barrier.
template <typename A, bool DELTA, int LANES, int CN>
struct ScanCfg {
  static constexpr int DP = LANES * 16;              // padded rows
  static constexpr int GW = 32 / LANES;              // column groups per warp
  static constexpr int CW = GW * CN;                 // columns per warp
  static constexpr int CT = 4 * CW;                  // columns per CTA
  static constexpr int TPL = RC / LANES;             // tokens whose sums a lane ends up with
  static constexpr int REC = Rec<DP, DELTA>::FLOATS;
  static constexpr int VN = (RC * CT + 127) / 128;
  static constexpr int SMEM = (2 * REC + 2 * RC * CT + (DELTA ? 2 * RC * CT : 0)) * 4 + 64;
};

template <typename A, bool DELTA, int LANES, int CN>
__global__ void __launch_bounds__(128) recur_scan_kernel(const ScanParams p) {
  using Cfg = ScanCfg<A, DELTA, LANES, CN>;
  constexpr int DP = Cfg::DP, CT = Cfg::CT, CW = Cfg::CW, REC = Cfg::REC, TPL = Cfg::TPL, VN = Cfg::VN;
  extern __shared__ __align__(128) float sm[];
  float* sV = sm + 2 * REC;                          // [2][RC][CT]
  float* sX = sV + 2 * RC * CT;                      // [RC][CT] per-warp column blocks: V - W, then U
  float* sU = sX + RC * CT;
  uint64_t* full = reinterpret_cast<uint64_t*>(sm + (Cfg::SMEM - 64) / 4);
  volatile int* s_abort = reinterpret_cast<volatile int*>(full + 2);
  const int seq = blockIdx.z, h = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rl = lane % LANES, cw = (lane / LANES) * CN, cloc = warp * CW + cw, c0 = blockIdx.x * CT;
  const int row0 = p.rv.cu[seq], len = p.rv.cu[seq + 1] - row0;
  if (len <= 0) return;
  const int ch0 = p.cv.first[seq], n_ch = (len + RC - 1) / RC;
  float* st = p.state + ((long long)p.rv.slot[seq] * p.H + h) * p.d * p.dv;
  const bool fresh = p.rv.pos0[seq] == 0;
  const float* rec = p.rec + ((long long)ch0 * p.H + h) * REC;
  const long long rec_step = (long long)p.H * REC;
  if (tid == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    *s_abort = 0;
    mbar_fence_init();
    mbar_expect_tx(&full[0], REC * 4);
    bulk_load(sm, rec, REC * 4, &full[0]);
  }
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
  float vreg[VN];
  auto load_v = [&](int t0) {
    const int nt = min(RC, len - t0);
#pragma unroll
    for (int n = 0; n < VN; ++n) {
      const int i = tid + n * 128, t = i / CT, c = c0 + i % CT;
      vreg[n] = (i < RC * CT && t < nt && c < p.dv)
                    ? to_f(reinterpret_cast<const A*>(p.v)[(long long)(row0 + t0 + t) * p.v_ld + (long long)h * p.dv + c])
                    : 0.f;
    }
  };
  auto put_v = [&](int buf) {
#pragma unroll
    for (int n = 0; n < VN; ++n) {
      const int i = tid + n * 128;
      if (i < RC * CT) sV[buf * RC * CT + i] = vreg[n];
    }
  };
  load_v(0);
  put_v(0);
  __syncthreads();
  // sum over this thread's rows of S[cn] * op[t][rows], for the 16 tokens, then over the lanes of the column
  using RL = Rec<DP, DELTA>;
  auto project = [&](const float* op, float (&acc)[CN][RC]) {
#pragma unroll
    for (int t = 0; t < RC; ++t) {
      u64 a[CN][2];
#pragma unroll
      for (int cn = 0; cn < CN; ++cn) a[cn][0] = a[cn][1] = 0;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(op + t * RL::LQ + c * LANES * 4 + rl * 4);
#pragma unroll
        for (int cn = 0; cn < CN; ++cn) {
          a[cn][0] = fma2(S[cn][2 * c], x.x, a[cn][0]);
          a[cn][1] = fma2(S[cn][2 * c + 1], x.y, a[cn][1]);
        }
      }
#pragma unroll
      for (int cn = 0; cn < CN; ++cn) {
        const float2 x = unpack2(a[cn][0]), y = unpack2(a[cn][1]);
        acc[cn][t] = (x.x + x.y) + (y.x + y.y);
      }
    }
#pragma unroll
    for (int cn = 0; cn < CN; ++cn) reduce_tokens<LANES>(acc[cn], rl);
  };
  bool ok = true;
  for (int ci = 0; ci < n_ch; ++ci) {
    const int buf = ci & 1, t0 = ci * RC, nt = min(RC, len - t0);
    if (ci + 1 < n_ch) {
      if (tid == 0) {
        mbar_expect_tx(&full[buf ^ 1], REC * 4);
        bulk_load(sm + (buf ^ 1) * REC, rec + (ci + 1) * rec_step, REC * 4, &full[buf ^ 1]);
      }
      load_v(t0 + RC);
    }
    ok = mbar_wait_warp(&full[buf], (ci >> 1) & 1, s_abort, p.status, ST_TIMEOUT_PRODUCER);
    if (!ok) break;
    const float* R = sm + buf * REC;
    const float* Kd = R + RL::KD;
    const float* Gl = R + RL::GL;
    const float* B = R + RL::B;
    const float* V = sV + buf * RC * CT;
    const float* U = V;
    if constexpr (DELTA) {
      float w[CN][RC];
      project(R + RL::GK, w);
#pragma unroll
      for (int i = 0; i < TPL; ++i)
#pragma unroll
        for (int cn = 0; cn < CN; ++cn) {
          const int t = rl * TPL + i;
          sX[t * CT + cloc + cn] = V[t * CT + cloc + cn] - w[cn][i];
        }
    }
    float q[CN][RC];
    project(R, q);
    if constexpr (DELTA) {
      __syncwarp();
      const float* Tm = R + RL::TM;
      float x[CN][TPL];
#pragma unroll
      for (int cn = 0; cn < CN; ++cn)
#pragma unroll
        for (int i = 0; i < TPL; ++i) x[cn][i] = 0.f;
#pragma unroll
      for (int j = 0; j < RC; j += 4) {
        float xv[CN][4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int cn = 0; cn < CN; ++cn) xv[cn][e] = sX[(j + e) * CT + cloc + cn];
#pragma unroll
        for (int i = 0; i < TPL; ++i) {
          const float4 m = *reinterpret_cast<const float4*>(Tm + (rl * TPL + i) * RL::LB + j);
#pragma unroll
          for (int cn = 0; cn < CN; ++cn)
            x[cn][i] = fmaf(m.w, xv[cn][3], fmaf(m.z, xv[cn][2], fmaf(m.y, xv[cn][1], fmaf(m.x, xv[cn][0], x[cn][i]))));
        }
      }
#pragma unroll
      for (int i = 0; i < TPL; ++i)
#pragma unroll
        for (int cn = 0; cn < CN; ++cn) sU[(rl * TPL + i) * CT + cloc + cn] = x[cn][i];
      __syncwarp();
      U = sU;
    }
    // read-out: the chunk's own writes join what the state held before it
#pragma unroll
    for (int j = 0; j < RC; j += 4) {
      float uv[CN][4];
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int cn = 0; cn < CN; ++cn) uv[cn][e] = U[(j + e) * CT + cloc + cn];
#pragma unroll
      for (int i = 0; i < TPL; ++i) {
        const float4 m = *reinterpret_cast<const float4*>(B + (rl * TPL + i) * RL::LB + j);
#pragma unroll
        for (int cn = 0; cn < CN; ++cn)
          q[cn][i] = fmaf(m.w, uv[cn][3], fmaf(m.z, uv[cn][2], fmaf(m.y, uv[cn][1], fmaf(m.x, uv[cn][0], q[cn][i]))));
      }
    }
#pragma unroll
    for (int i = 0; i < TPL; ++i) {
      const int t = rl * TPL + i;
#pragma unroll
      for (int cn = 0; cn < CN; ++cn)
        if (t < nt && c0 + cloc + cn < p.dv) p.o[((long long)(row0 + t0 + t) * p.H + h) * p.dv + c0 + cloc + cn] = q[cn][i];
    }
    // state behind the chunk
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(Gl + c * LANES * 4 + rl * 4);
#pragma unroll
      for (int cn = 0; cn < CN; ++cn) {
        S[cn][2 * c] = mul2(S[cn][2 * c], g.x);
        S[cn][2 * c + 1] = mul2(S[cn][2 * c + 1], g.y);
      }
    }
#pragma unroll
    for (int t = 0; t < RC; ++t) {
      u64 u2[CN];
#pragma unroll
      for (int cn = 0; cn < CN; ++cn) {
        const float x = U[t * CT + cloc + cn];
        u2[cn] = pack2(x, x);
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(Kd + t * RL::LK + c * LANES * 4 + rl * 4);
#pragma unroll
        for (int cn = 0; cn < CN; ++cn) {
          S[cn][2 * c] = fma2(k.x, u2[cn], S[cn][2 * c]);
          S[cn][2 * c + 1] = fma2(k.y, u2[cn], S[cn][2 * c + 1]);
        }
      }
    }
    if (ci + 1 < n_ch) put_v(buf ^ 1);
    __syncthreads();
  }
  if (*s_abort) {
    bounded_delay_ns(2000000);
    return;
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

// ------------------------------------------------------------------ the same scan on tensor cores
// All products of a chunk are small matrix products with the transposed state S^T [columns, d] as an operand or result:
//   W^T = S^T (G k)^T, Q^T = S^T (G q)^T,  U^T = (V - W)^T Tm^T,  O^T = Q^T + U^T B^T,  S^T <- S^T G_last + U^T Kd
// They run as mma.m16n8k8 with every fp32 operand split into two TF32 terms (x = hi + lo with lo = x - hi exactly) and three
// products hi hi + hi lo + lo hi accumulated in fp32: what is dropped, lo lo and the rounding of lo, is below 2^-21 of a
// product. The accumulator layout of m16n8 (columns 2t, 2t + 1 of row g) is read back as an A operand whose k index t / t + 4
// stands for 2t / 2t + 1; the B operands are fetched in that order, so state, W, Q, U and O never leave their registers.
// A warp owns 16 value columns. SPLITD: the four warps of a CTA share those columns and own a quarter of d each (few
// sequences: more CTAs); otherwise they own 16 columns each.
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi));
}
// accumulator fragment -> A operand terms
__device__ __forceinline__ void split_frag(const float (&c)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  split_tf32(c[0], hi[0], lo[0]);
  split_tf32(c[2], hi[1], lo[1]);
  split_tf32(c[1], hi[2], lo[2]);
  split_tf32(c[3], hi[3], lo[3]);
}
// The three products of a split pair in accumulators of their own (short dependency chains), summed by the caller.
__device__ __forceinline__ void mma_split3(float (&c)[3][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], float b0, float b1) {
  uint32_t h0, l0, h1, l1;
  split_tf32(b0, h0, l0);
  split_tf32(b1, h1, l1);
  mma_tf32(c[0], ah, h0, h1);
  mma_tf32(c[1], ah, l0, l1);
  mma_tf32(c[2], al, h0, h1);
}
template <bool A_EXACT>
__device__ __forceinline__ void mma_split(float (&c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], float b0, float b1) {
  uint32_t h0, l0, h1, l1;
  split_tf32(b0, h0, l0);
  split_tf32(b1, h1, l1);
  mma_tf32(c, ah, l0, l1);
  if (!A_EXACT) mma_tf32(c, al, h0, h1);
  mma_tf32(c, ah, h0, h1);
}

template <bool DELTA, int DP, bool SPLITD>
struct TcScanCfg {
  static constexpr int COLS = SPLITD ? 16 : 64;
  static constexpr int ND = (SPLITD ? DP / 4 : DP) / 8;       // 8-row tiles of d per warp
  static constexpr int REC = Rec<DP, DELTA>::FLOATS;
  static constexpr int XCH = SPLITD ? 2 * 4 * (1 + DELTA) * 8 * 32 : 0;   // [2][warp][quantity][8 values][lane]
  static constexpr int FIT = (227 * 256 - 16 - XCH) / REC;
  static constexpr int WANT = SPLITD ? 4 : (DELTA ? 2 : 3);   // the larger records leave room for more CTAs with two
  static constexpr int STAGES = FIT < WANT ? FIT : WANT;
  static constexpr int SMEM = (STAGES * REC + XCH) * 4 + 64;
  static_assert(STAGES >= 2 && SMEM <= 227 * 1024, "shared memory");
};

template <typename A, bool DELTA, int DP, bool SPLITD>
__global__ void __launch_bounds__(128) recur_scan_tc_kernel(const ScanParams p) {
  using Cfg = TcScanCfg<DELTA, DP, SPLITD>;
  using RL = Rec<DP, DELTA>;
  constexpr int ND = Cfg::ND, REC = Cfg::REC, STAGES = Cfg::STAGES;
  constexpr bool V_EXACT = !DELTA && sizeof(A) == 2;          // bf16 values have no low TF32 term
  extern __shared__ __align__(128) float sm[];
  float* xch = sm + STAGES * REC;
  uint64_t* full = reinterpret_cast<uint64_t*>(sm + (Cfg::SMEM - 64) / 4);
  volatile int* s_abort = reinterpret_cast<volatile int*>(full + STAGES);
  const int seq = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int c0 = blockIdx.x * Cfg::COLS + (SPLITD ? 0 : warp * 16), d0 = SPLITD ? warp * (DP / 4) : 0;
  const int row0 = p.rv.cu[seq], len = p.rv.cu[seq + 1] - row0;
  if (len <= 0) return;
  const int n_ch = (len + RC - 1) / RC;
  float* st = p.state + ((long long)p.rv.slot[seq] * p.H + h) * p.d * p.dv;
  const bool fresh = p.rv.pos0[seq] == 0;
  const float* rec = p.rec + ((long long)p.cv.first[seq] * p.H + h) * REC;
  const long long rec_step = (long long)p.H * REC;
  if (tid == 0) {
    for (int s = 0; s < STAGES; ++s) mbar_init(&full[s], 1);
    *s_abort = 0;
    mbar_fence_init();
    for (int s = 0; s < STAGES && s < n_ch; ++s) {
      mbar_expect_tx(&full[s], REC * 4);
      bulk_load(sm + s * REC, rec + s * rec_step, REC * 4, &full[s]);
    }
  }
  float S[ND][4];
#pragma unroll
  for (int j = 0; j < ND; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = d0 + 8 * j + 2 * t + (e & 1), c = c0 + g + (e >> 1) * 8;
      S[j][e] = (!fresh && r < p.d && c < p.dv) ? st[(long long)r * p.dv + c] : 0.f;
    }
  // values of a chunk in accumulator layout: token 8 n + 2 t + (e & 1), column g + 8 (e >> 1)
  const A* vp = reinterpret_cast<const A*>(p.v) + (long long)h * p.dv;
  // (kept as loaded until the next chunk converts them: a conversion here would wait for the load)
  auto load_v = [&](int t0, A (&v)[2][4]) {
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int tok = t0 + 8 * n + 2 * t + (e & 1), c = c0 + g + (e >> 1) * 8;
        v[n][e] = from_f<A>(0.f);
        if (tok < len && c < p.dv) v[n][e] = vp[(long long)(row0 + tok) * p.v_ld + c];
      }
  };
  A vn[2][4];
  load_v(0, vn);
  __syncthreads();
  for (int ci = 0; ci < n_ch; ++ci) {
    const int buf = ci % STAGES, t0 = ci * RC;
    float v[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) v[n][e] = to_f(vn[n][e]);
    if (ci + 1 < n_ch) load_v(t0 + RC, vn);
    if (!mbar_wait_warp(&full[buf], (ci / STAGES) & 1, s_abort, p.status, ST_TIMEOUT_PRODUCER)) break;
    const float* R = sm + buf * REC;
    float q[2][4], w[2][4];
    {
      float q3[2][3][4], w3[2][3][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int x = 0; x < 3; ++x)
#pragma unroll
          for (int e = 0; e < 4; ++e) q3[n][x][e] = w3[n][x][e] = 0.f;
#pragma unroll
      for (int j = 0; j < ND; ++j) {
        uint32_t ah[4], al[4];
        split_frag(S[j], ah, al);
        const float* base = R + g * RL::LQ + d0 + 8 * j + 2 * t;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          if constexpr (DELTA) {
            const float2 b = *reinterpret_cast<const float2*>(base + RL::GK + n * 8 * RL::LQ);
            mma_split3(w3[n], ah, al, b.x, b.y);
          }
          const float2 b = *reinterpret_cast<const float2*>(base + n * 8 * RL::LQ);
          mma_split3(q3[n], ah, al, b.x, b.y);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          q[n][e] = q3[n][0][e] + (q3[n][1][e] + q3[n][2][e]);
          w[n][e] = w3[n][0][e] + (w3[n][1][e] + w3[n][2][e]);
        }
    }
    if constexpr (SPLITD) {
      float* x = xch + (ci & 1) * 4 * (1 + DELTA) * 256;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          x[(warp * (1 + DELTA)) * 256 + (n * 4 + e) * 32 + lane] = q[n][e];
          if (DELTA) x[(warp * 2 + 1) * 256 + (n * 4 + e) * 32 + lane] = w[n][e];
        }
      __syncthreads();
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = (n * 4 + e) * 32 + lane;
          q[n][e] = (x[i] + x[(1 + DELTA) * 256 + i]) + (x[2 * (1 + DELTA) * 256 + i] + x[3 * (1 + DELTA) * 256 + i]);
          if (DELTA) w[n][e] = (x[256 + i] + x[768 + i]) + (x[1280 + i] + x[1792 + i]);
        }
    }
    uint32_t uh[2][4], ul[2][4];       // written values as A operand
    if constexpr (DELTA) {
      float u[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          w[n][e] = v[n][e] - w[n][e];
          u[n][e] = 0.f;
        }
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        uint32_t xh[4], xl[4];
        split_frag(w[k], xh, xl);
#pragma unroll
        for (int n = 0; n < 2; ++n)
          if (k <= n) {                // lower triangular
            const float2 b = *reinterpret_cast<const float2*>(R + RL::TM + (n * 8 + g) * RL::LB + k * 8 + 2 * t);
            mma_split<false>(u[n], xh, xl, b.x, b.y);
          }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) split_frag(u[n], uh[n], ul[n]);
    } else {
#pragma unroll
      for (int n = 0; n < 2; ++n) split_frag(v[n], uh[n], ul[n]);
    }
    if (!SPLITD || warp == (ci & 3)) {
#pragma unroll
      for (int k = 0; k < 2; ++k)
#pragma unroll
        for (int n = 0; n < 2; ++n)
          if (k <= n) {
            const float2 b = *reinterpret_cast<const float2*>(R + RL::B + (n * 8 + g) * RL::LB + k * 8 + 2 * t);
            mma_split<V_EXACT>(q[n], uh[k], ul[k], b.x, b.y);
          }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int tok = t0 + 8 * n + 2 * t + (e & 1), c = c0 + g + (e >> 1) * 8;
          if (tok < len && c < p.dv) p.o[((long long)(row0 + tok) * p.H + h) * p.dv + c] = q[n][e];
        }
    }
#pragma unroll
    for (int j = 0; j < ND; ++j) {
      const float2 gl = *reinterpret_cast<const float2*>(R + RL::GL + d0 + 8 * j + 2 * t);
      S[j][0] *= gl.x; S[j][1] *= gl.y; S[j][2] *= gl.x; S[j][3] *= gl.y;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const float* kd = R + RL::KD + (k * 8 + 2 * t) * RL::LK + d0 + 8 * j + g;
        mma_split<V_EXACT>(S[j], uh[k], ul[k], kd[0], kd[RL::LK]);
      }
    }
    __syncthreads();
    if (tid == 0 && ci + STAGES < n_ch) {
      mbar_expect_tx(&full[buf], REC * 4);
      bulk_load(sm + buf * REC, rec + (ci + STAGES) * rec_step, REC * 4, &full[buf]);
    }
  }
  if (*s_abort) {
    bounded_delay_ns(2000000);
    return;
  }
#pragma unroll
  for (int j = 0; j < ND; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = d0 + 8 * j + 2 * t + (e & 1), c = c0 + g + (e >> 1) * 8;
      if (r < p.d && c < p.dv) st[(long long)r * p.dv + c] = S[j][e];
    }
}

// ------------------------------------------------------------------ one token per sequence
// One CTA per (head, sequence): operands from the projected rows (convolution, unit norms, gates), one state update with
// the state tile in registers between its two passes, read-out, per-head norm and output gate.
struct StepParams {
  DeltaParams in;             // delta rule: projected rows and constants (v unused)
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
__global__ void __launch_bounds__(256, NR <= 16 ? 2 : 1) recur_step_kernel(const StepParams p) {
  extern __shared__ __align__(128) float sm[];
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
  const int lpr = p.lpr, RG = 256 / lpr, rg = tid / lpr, cl = tid % lpr;
  float* st = p.state + ((long long)slot * p.H + h) * p.d * p.dv;
  const bool fresh = pos == 0;
  float S[NR][VEC];
  auto load_state = [&](int col) {
#pragma unroll
    for (int n = 0; n < NR; ++n) {
      const int r = rg + n * RG;
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[n][e] = 0.f;
      if (!fresh && col < p.dv && r < p.d) {
        if constexpr (VEC == 4) {
          const float4 x = *reinterpret_cast<const float4*>(st + (long long)r * p.dv + col);
          S[n][0] = x.x; S[n][1] = x.y; S[n][2] = x.z; S[n][3] = x.w;
        } else {
          S[n][0] = st[(long long)r * p.dv + col];
        }
      }
    }
  };
  load_state(cl * VEC);       // in flight while the operands are prepared
  float beta = 0.f;
  if constexpr (DELTA) {
    const DeltaParams& in = p.in;
    const int C = 2 * in.G * in.d + in.H * in.dv;
    const A* row = reinterpret_cast<const A*>(in.u) + (long long)t * in.u_ld;
    A* ring = reinterpret_cast<A*>(in.ring) + (long long)slot * in.taps * C;
    A* e = ring + (long long)(pos % in.taps) * C;     // the entry this token fills; no head reads it in this step
    const bool owner = h % (p.H / p.Hq) == 0;
    for (int i = tid; i < 2 * in.d + in.dv; i += 256) {
      const bool is_v = i >= 2 * in.d;
      const int which = i / in.d, c = is_v ? i - 2 * in.d : i % in.d;
      const int col = is_v ? 2 * in.G * in.d + h * in.dv + c : (which * in.G + hq) * in.d + c;
      float y[1];
      conv_walk<A, 1, 8>(row, in.u_ld, in.wconv, in.taps, C, col, ring, pos, 0, 1, y);
      const float x = y[0] * sigmoid_f(y[0]);
      if (is_v) sv[c] = to_f(from_f<A>(x));
      else (which ? sk : sq)[c] = x;
      if (in.taps > 1 && (is_v || owner)) e[col] = row[col];
    }
    const A* ar = reinterpret_cast<const A*>(in.a) + (long long)t * in.a_ld + (long long)h * in.d;
    const float al = -expf(in.a_log[h]);
    for (int i = tid; i < in.d; i += 256) sg[i] = expf(al * softplus_f(to_f(ar[i]) + in.dt_bias[h * in.d + i]));
    beta = sigmoid_f(to_f(reinterpret_cast<const A*>(in.b)[(long long)t * in.b_ld + h]));
    __syncthreads();
    if (warp < 2) {           // unit norms; the query also takes d^-1/2
      float* x = warp ? sk : sq;
      float ss = 0.f;
      for (int i = lane; i < in.d; i += 32) ss += x[i] * x[i];
      ss = warp_sum(ss);
      const float r = (warp ? 1.f : 1.f / sqrtf((float)in.d)) / sqrtf(ss + 1e-6f);
      for (int i = lane; i < in.d; i += 32) x[i] *= r;
    }
  } else {
    const A* qr = reinterpret_cast<const A*>(p.qr) + (long long)t * p.ld + (long long)h * p.d;
    const A* fr = reinterpret_cast<const A*>(p.fr) + (long long)t * p.ld + (long long)h * p.d;
    const A* vr = reinterpret_cast<const A*>(p.vr) + (long long)t * p.ld + (long long)h * p.dv;
    for (int i = tid; i < p.d + p.dv; i += 256) {
      if (i < p.d) {
        const float z = to_f(qr[i]);
        sq[i] = z * sigmoid_f(z);
        const float l = p.lower[h * p.d + i];
        const float f = l + (1.f - l) * sigmoid_f(to_f(fr[i]) + p.fbias[h * p.d + i]);
        sg[i] = f;
        sk[i] = 1.f - f;
      } else {
        sv[i - p.d] = to_f(vr[i - p.d]);
      }
    }
  }
  __syncthreads();

  for (int ct = 0; ct < p.dv; ct += lpr * VEC) {
    const int col = ct + cl * VEC;
    const bool on = col < p.dv;
    if (ct) load_state(col);
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
  p->a_log = a->a_log; p->dt_bias = a->dt_bias; p->v = a->v;
  p->rv = view(&a->ragged);
  p->T = a->T; p->H = a->H; p->G = a->G; p->d = a->d; p->dv = a->dv; p->taps = a->taps;
}
static int pad_rows(int d) { return d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256; }

// Floats of scratch that the records of one (chunk, head) take.
extern "C" int sx_recur_record(int d, int delta) {
  switch (pad_rows(d)) {
    case 32: return delta ? Rec<32, true>::FLOATS : Rec<32, false>::FLOATS;
    case 64: return delta ? Rec<64, true>::FLOATS : Rec<64, false>::FLOATS;
    case 128: return delta ? Rec<128, true>::FLOATS : Rec<128, false>::FLOATS;
    default: return delta ? Rec<256, true>::FLOATS : Rec<256, false>::FLOATS;
  }
}

template <typename K>
static int allow_smem(K kern, int bytes, bool* done) {
  if (!*done && bytes > 48 * 1024) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) != cudaSuccess) return -10;
    *done = true;
  }
  return 0;
}

template <typename A, int DP>
static int launch_gate_chunks(const SxGateArgs* a, cudaStream_t st) {
  static bool set = false;
  const int smem = 3 * RC * DP * 4;
  if (int rc = allow_smem(gate_chunk_kernel<A, DP>, smem, &set)) return rc;
  gate_chunk_kernel<A, DP><<<dim3(a->chunks.n, a->H), 256, smem, st>>>((const A*)a->q, (const A*)a->f, a->ld, a->bias, a->lower, a->rec,
                                                                       view(&a->ragged), chunks(&a->chunks), a->H, a->d);
  return last_rc();
}

// Records of the gated-write recurrence from projected rows (q and forget-gate logits).
extern "C" int sx_gate_chunks(const SxGateArgs* a, cudaStream_t st) {
  if (a->chunks.n <= 0) return 0;
  if (a->d <= 0 || a->d > 256) return -1;
  SX_ACT_DISPATCH(a->f32, {
    switch (pad_rows(a->d)) {
      case 32: return launch_gate_chunks<A, 32>(a, st);
      case 64: return launch_gate_chunks<A, 64>(a, st);
      case 128: return launch_gate_chunks<A, 128>(a, st);
      default: return launch_gate_chunks<A, 256>(a, st);
    }
  });
  return 0;
}

template <typename A, int DP>
static int launch_ssd_chunks(const SxSsdArgs* a, float* rec, cudaStream_t st) {
  static bool set = false;
  const int smem = 3 * RC * DP * 4;
  if (int rc = allow_smem(ssd_chunk_kernel<A, DP>, smem, &set)) return rc;
  ssd_chunk_kernel<A, DP><<<dim3(a->chunks.n, a->H), 256, smem, st>>>((const A*)a->b, (const A*)a->c, a->dt, a->la, rec, view(&a->ragged),
                                                                      chunks(&a->chunks), a->H, a->G, a->N, a->np);
  return last_rc();
}

// Records of the SSD recurrence from its operands.
extern "C" int sx_ssd_chunks(const SxSsdArgs* a, float* rec, cudaStream_t st) {
  if (a->chunks.n <= 0) return 0;
  if (a->N <= 0 || a->N > 256 || a->G <= 0 || a->H % a->G) return -1;
  SX_ACT_DISPATCH(a->f32, {
    switch (pad_rows(a->N)) {
      case 32: return launch_ssd_chunks<A, 32>(a, rec, st);
      case 64: return launch_ssd_chunks<A, 64>(a, rec, st);
      case 128: return launch_ssd_chunks<A, 128>(a, rec, st);
      default: return launch_ssd_chunks<A, 256>(a, rec, st);
    }
  });
  return 0;
}

template <typename A, int DP, int MT>
static int launch_delta_chunks(const DeltaParams& p, float* rec, const ChunkView& cv, cudaStream_t st) {
  static bool set = false;
  const int smem = (3 * RC * DP + RC * RC + RC) * 4;
  if (int rc = allow_smem(delta_chunk_kernel<A, DP, MT>, smem, &set)) return rc;
  delta_chunk_kernel<A, DP, MT><<<dim3(cv.n_chunks, p.H), 256, smem, st>>>(p, rec, cv);
  return last_rc();
}
template <typename A, int DP>
static int pick_delta_chunks(const DeltaParams& p, float* rec, const ChunkView& cv, cudaStream_t st) {
  return p.taps <= 4 ? launch_delta_chunks<A, DP, 4>(p, rec, cv, st) : launch_delta_chunks<A, DP, 8>(p, rec, cv, st);
}

// Records and convolved values of the gated delta rule from projected rows.
extern "C" int sx_delta_chunks(const SxDeltaArgs* a, const SxChunks* c, float* rec, cudaStream_t st) {
  if (c->n <= 0) return 0;
  if (a->d <= 0 || a->d > 256 || a->G <= 0 || a->H % a->G || a->taps < 1 || a->taps > 8) return -1;
  DeltaParams p;
  fill_delta(&p, a);
  const ChunkView cv = chunks(c);
  SX_ACT_DISPATCH(a->f32, {
    switch (pad_rows(a->d)) {
      case 32: return pick_delta_chunks<A, 32>(p, rec, cv, st);
      case 64: return pick_delta_chunks<A, 64>(p, rec, cv, st);
      case 128: return pick_delta_chunks<A, 128>(p, rec, cv, st);
      default: return pick_delta_chunks<A, 256>(p, rec, cv, st);
    }
  });
  return 0;
}

template <typename A, bool DELTA, int LANES, int CN>
static int launch_scan(const ScanParams& p, cudaStream_t st) {
  using Cfg = ScanCfg<A, DELTA, LANES, CN>;
  static bool set = false;
  if (int rc = allow_smem(recur_scan_kernel<A, DELTA, LANES, CN>, Cfg::SMEM, &set)) return rc;
  dim3 grid((p.dv + Cfg::CT - 1) / Cfg::CT, p.H, p.rv.n);
  recur_scan_kernel<A, DELTA, LANES, CN><<<grid, 128, Cfg::SMEM, st>>>(p);
  return last_rc();
}
template <typename A, bool DELTA>
static int pick_scan(const ScanParams& p, cudaStream_t st) {
  // two columns per thread once one column per thread would put more than two CTAs on every SM
  const int lanes = pad_rows(p.d) / 16, ct1 = 4 * (32 / lanes);
  const bool wide = (long long)((p.dv + ct1 - 1) / ct1) * p.H * p.rv.n > 2 * 148;
#define SX_SCAN(L) return wide ? launch_scan<A, DELTA, L, 2>(p, st) : launch_scan<A, DELTA, L, 1>(p, st)
  switch (lanes) {
    case 2: SX_SCAN(2);
    case 4: SX_SCAN(4);
    case 8: SX_SCAN(8);
    default: SX_SCAN(16);
  }
#undef SX_SCAN
}

template <typename A, bool DELTA, int DP, bool SPLITD>
static int launch_scan_tc(const ScanParams& p, cudaStream_t st) {
  using Cfg = TcScanCfg<DELTA, DP, SPLITD>;
  static bool set = false;
  if (int rc = allow_smem(recur_scan_tc_kernel<A, DELTA, DP, SPLITD>, Cfg::SMEM, &set)) return rc;
  dim3 grid((p.dv + Cfg::COLS - 1) / Cfg::COLS, p.H, p.rv.n);
  recur_scan_tc_kernel<A, DELTA, DP, SPLITD><<<grid, 128, Cfg::SMEM, st>>>(p);
  return last_rc();
}
template <bool DELTA>
static int pick_scan_tc(const ScanParams& p, cudaStream_t st) {
  using A = __nv_bfloat16;
  const bool many = (long long)((p.dv + 63) / 64) * p.H * p.rv.n >= 148;   // 64 columns per CTA already fill the machine
#define SX_SCAN_TC(D) return many ? launch_scan_tc<A, DELTA, D, false>(p, st) : launch_scan_tc<A, DELTA, D, true>(p, st)
  switch (pad_rows(p.d)) {
    case 32: SX_SCAN_TC(32);
    case 64: SX_SCAN_TC(64);
    case 128: SX_SCAN_TC(128);
    default: SX_SCAN_TC(256);
  }
#undef SX_SCAN_TC
}

// delta != 0: gated delta rule; else the gated write. Portions are independent of each other. 32-bit runs take the SIMT
// kernel, bf16 runs the tensor-core kernel.
extern "C" int sx_recur_scan(const SxScanArgs* a, cudaStream_t st) {
  if (a->ragged.n <= 0) return 0;
  if (a->d <= 0 || a->d > 256 || a->dv <= 0) return -1;
  ScanParams p;
  p.rec = a->rec; p.v = a->v; p.v_ld = a->v_ld; p.state = a->state; p.o = a->o; p.status = a->status;
  p.rv = view(&a->ragged); p.cv = chunks(&a->chunks);
  p.H = a->H; p.d = a->d; p.dv = a->dv;
  if (a->f32) return a->delta ? pick_scan<float, true>(p, st) : pick_scan<float, false>(p, st);
  return a->delta ? pick_scan_tc<true>(p, st) : pick_scan_tc<false>(p, st);
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
  if (a->d <= 0 || a->d > 256 || a->dv <= 0 || a->Hq <= 0 || a->H % a->Hq || (a->delta && (a->in.taps < 1 || a->in.taps > 8))) return -1;
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
