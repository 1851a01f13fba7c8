// SSD (Mamba-2) recurrence for serving: ragged portions from any stored state, fp32 state [slots, H, N, P] per head.
//   S <- exp(-exp(A_log) dt) S + dt B x^T,   y = (S^T C + D x) silu(z),   head h reads B and C of group h / (H / G)
// Operands for the prompt forms, the output gate of 32-bit prompts, and the one-token step of decoding. The state and
// everything that enters it besides the convolved projections is fp32.
#include "common.cuh"
#include "ragged.cuh"
#include "sx_api.h"

namespace sx {

struct SsdParams {
  SxSsdArgs a;
  RaggedView rv;
  ChunkView cv;
};

// ------------------------------------------------------------------ operands: convolution, step sizes, decays
// A thread walks one column of the operand layout [x: H xp | B: G np | C: G np | dt: H] through the 16 rows of a chunk.
template <typename A, int MT>
__global__ void __launch_bounds__(256) ssd_operands_kernel(const SsdParams P) {
  const SxSsdArgs& p = P.a;
  const int ch = blockIdx.y, seq = P.cv.seq[ch], s0 = P.cv.start[ch];
  const int row0 = P.rv.cu[seq] + s0, nt = min(RC, P.rv.cu[seq + 1] - row0), pos = P.rv.pos0[seq] + s0;
  const int inner = p.H * p.P, C = inner + 2 * p.G * p.N, wx = p.H * p.xp, wn = p.G * p.np;
  const int i = blockIdx.x * 256 + threadIdx.x;
  const A* u = reinterpret_cast<const A*>(p.u) + (long long)row0 * p.u_ld;
  if (i >= wx + 2 * wn) {
    const int h = i - wx - 2 * wn;
    if (h >= p.H) return;
    const float al = -expf(p.a_log[h]), bias = p.dt_bias[h];
    for (int t = 0; t < nt; ++t) {
      const float dt = softplus_f(to_f(u[(long long)t * p.u_ld + inner + C + h]) + bias);
      p.dt[(long long)(row0 + t) * p.H + h] = dt;
      p.la[(long long)(row0 + t) * p.H + h] = al * dt;
    }
    return;
  }
  int col, ld;          // convolution channel (or -1: padding), output pitch
  A* out;
  if (i < wx) {
    col = i % p.xp < p.P ? i / p.xp * p.P + i % p.xp : -1;
    out = reinterpret_cast<A*>(p.x) + i;
    ld = wx;
  } else {
    const int j = (i - wx) % wn, which = (i - wx) / wn;
    col = j % p.np < p.N ? inner + (which * p.G + j / p.np) * p.N + j % p.np : -1;
    out = reinterpret_cast<A*>(which ? p.c : p.b) + j;
    ld = wn;
  }
  out += (long long)row0 * ld;
  float y[RC];
  if (col >= 0) {
    const A* ring = reinterpret_cast<const A*>(p.ring) + (long long)P.rv.slot[seq] * p.taps * C;
    conv_walk<A, RC, MT>(u + inner, p.u_ld, p.wconv, p.taps, C, col, ring, pos, s0, nt, y);
    const float b = p.bconv[col];
#pragma unroll
    for (int t = 0; t < RC; ++t) y[t] = silu_act<A>(y[t] + b);
  } else {
#pragma unroll
    for (int t = 0; t < RC; ++t) y[t] = 0.f;
  }
#pragma unroll
  for (int t = 0; t < RC; ++t)
    if (t < nt) out[(long long)t * ld] = from_f<A>(y[t]);
}

// ------------------------------------------------------------------ skip connection and output gate
template <typename A>
__global__ void __launch_bounds__(256) ssd_gate_kernel(const SsdParams P, const float* __restrict__ o) {
  const SxSsdArgs& p = P.a;
  const int t = blockIdx.x, inner = p.H * p.P;
  const A* z = reinterpret_cast<const A*>(p.u) + (long long)t * p.u_ld;
  const A* x = reinterpret_cast<const A*>(p.x) + (long long)t * p.H * p.xp;
  A* y = reinterpret_cast<A*>(p.y) + (long long)t * p.y_ld;
  for (int i = threadIdx.x; i < inner; i += 256) {
    const int h = i / p.P;
    const float v = fmaf(p.D[h], to_f(x[h * p.xp + i - h * p.P]), o[(long long)t * inner + i]);
    y[i] = from_f<A>(v * silu_act<A>(to_f(z[i])));
  }
}

// ------------------------------------------------------------------ one token per sequence
// One CTA per (head, sequence). Threads own VEC columns of the state and walk its rows; the rows of a warp are summed by
// shuffles, the warps through shared memory.
template <typename A, int VEC>
__global__ void __launch_bounds__(256, 3) ssd_step_kernel(const SsdParams P, int lpr) {
  const SxSsdArgs& p = P.a;
  extern __shared__ __align__(16) float sm[];
  const int N = p.N, W = p.P;
  float* sB = sm;                 // [N] dt B
  float* sC = sB + N;             // [N]
  float* sx = sC + N;             // [W]
  float* red = sx + W;            // [8 warps][lpr * VEC]
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int slot = P.rv.slot[seq];
  if (slot < 0) return;           // padding row of a captured launch
  const int row = P.rv.cu[seq], pos = P.rv.pos0[seq], rep = p.H / p.G, g = h / rep;
  const int inner = p.H * W, C = inner + 2 * p.G * N;
  const A* u = reinterpret_cast<const A*>(p.u) + (long long)row * p.u_ld;
  A* ring = reinterpret_cast<A*>(p.ring) + (long long)slot * p.taps * C;
  const float dt = softplus_f(to_f(u[inner + C + h]) + p.dt_bias[h]);
  const float decay = pos == 0 ? 0.f : expf(-expf(p.a_log[h]) * dt);
  const int rows = 256 / lpr, r0 = tid / lpr, cv = W / VEC;
  float* st = p.state + ((long long)slot * p.H + h) * N * W;
  float S[8][VEC];
  auto load = [&](int c, int n0) {        // up to 8 rows of the state, all loads in flight together
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const int n = n0 + k * rows;
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[k][e] = 0.f;
      if (c < cv && n < N && pos != 0) {
        const float* s = st + (long long)n * W + c * VEC;
        if constexpr (VEC == 4) {
          const float4 v = __ldcs(reinterpret_cast<const float4*>(s));
          S[k][0] = v.x; S[k][1] = v.y; S[k][2] = v.z; S[k][3] = v.w;
        } else {
          S[k][0] = *s;
        }
      }
    }
  };
  load(tid % lpr, r0);                    // arrives while the convolutions run
  for (int i = tid; i < W + 2 * N; i += 256) {
    const int which = i < W ? 0 : (i - W) / N, n = i < W ? i : (i - W) % N;
    const int col = i < W ? h * W + i : inner + (which * p.G + g) * N + n;
    float y[1];
    conv_walk<A, 1, 8>(u + inner, p.u_ld, p.wconv, p.taps, C, col, ring, pos, 0, 1, y);
    // the entry written is not one that this step reads; heads of a group share B and C, their first one keeps them
    if (p.taps > 1 && (i < W || h % rep == 0)) ring[(long long)(pos % p.taps) * C + col] = u[inner + col];
    const float v = silu_act<A>(y[0] + p.bconv[col]);
    if (i < W) sx[i] = v;
    else if (which == 0) sB[n] = v * dt;
    else sC[n] = v;
  }
  __syncthreads();
  const A* z = u + (long long)h * W;
  A* out = reinterpret_cast<A*>(p.y) + (long long)row * p.y_ld + (long long)h * W;
  for (int cb = 0; cb < cv; cb += lpr) {
    const int c = cb + tid % lpr;
    const bool ok = c < cv;
    float acc[VEC], xv[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      acc[e] = 0.f;
      xv[e] = ok ? sx[c * VEC + e] : 0.f;
    }
    for (int n0 = r0; n0 < N; n0 += 8 * rows) {
      if (cb > 0 || n0 > r0) load(c, n0);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int n = n0 + k * rows;
        if (!ok || n >= N) continue;
        const float b = sB[n], cc = sC[n];
        float* s = st + (long long)n * W + c * VEC;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          S[k][e] = fmaf(decay, S[k][e], b * xv[e]);
          acc[e] = fmaf(cc, S[k][e], acc[e]);
        }
        if constexpr (VEC == 4) __stcs(reinterpret_cast<float4*>(s), make_float4(S[k][0], S[k][1], S[k][2], S[k][3]));
        else *s = S[k][0];
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e)
      for (int m = lpr; m < 32; m <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], m);
    __syncthreads();
    if (lane < lpr)
#pragma unroll
      for (int e = 0; e < VEC; ++e) red[(warp * lpr + lane) * VEC + e] = acc[e];
    __syncthreads();
    for (int i = tid; i < lpr * VEC; i += 256) {
      const int col = cb * VEC + i;
      if (col >= W) continue;
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) v += red[w * lpr * VEC + i];
      v = fmaf(p.D[h], sx[col], v);
      out[col] = from_f<A>(v * silu_act<A>(to_f(z[col])));
    }
  }
}

}  // namespace sx
using namespace sx;

static bool ssd_sizes(const SxSsdArgs* a) {
  return a->H > 0 && a->P > 0 && a->N > 0 && a->G > 0 && a->H % a->G == 0 && a->taps >= 1 && a->taps <= 8;
}
static SsdParams ssd_params(const SxSsdArgs* a) { return SsdParams{*a, view(&a->ragged), chunks(&a->chunks)}; }

extern "C" int sx_ssd_operands(const SxSsdArgs* a, cudaStream_t st) {
  if (a->chunks.n <= 0) return 0;
  if (!ssd_sizes(a) || a->xp < a->P || a->np < a->N) return -1;
  const SsdParams p = ssd_params(a);
  const dim3 grid((a->H * a->xp + 2 * a->G * a->np + a->H + 255) / 256, a->chunks.n);
  if (grid.y > 65535) return -2;
  SX_ACT_DISPATCH(a->f32, {
    if (a->taps <= 4) ssd_operands_kernel<A, 4><<<grid, 256, 0, st>>>(p);
    else ssd_operands_kernel<A, 8><<<grid, 256, 0, st>>>(p);
  });
  return last_rc();
}

extern "C" int sx_ssd_gate(const SxSsdArgs* a, const float* o, cudaStream_t st) {
  if (a->T <= 0) return 0;
  if (!ssd_sizes(a)) return -1;
  const SsdParams p = ssd_params(a);
  SX_ACT_DISPATCH(a->f32, (ssd_gate_kernel<A><<<a->T, 256, 0, st>>>(p, o)));
  return last_rc();
}

extern "C" int sx_ssd_step(const SxSsdArgs* a, cudaStream_t st) {
  if (a->ragged.n <= 0) return 0;
  if (!ssd_sizes(a) || a->ragged.n > 65535) return -1;
  const SsdParams p = ssd_params(a);
  const int vec = a->P % 4 == 0 ? 4 : 1, cv = a->P / vec;
  int lpr = 1;
  while (lpr < 32 && lpr < cv) lpr *= 2;
  const int smem = (2 * a->N + a->P + 8 * lpr * vec) * 4;
  if (smem > 48 * 1024) return -2;
  const dim3 grid(a->H, a->ragged.n);
  SX_ACT_DISPATCH(a->f32, {
    if (vec == 4) ssd_step_kernel<A, 4><<<grid, 256, smem, st>>>(p, lpr);
    else ssd_step_kernel<A, 1><<<grid, 256, smem, st>>>(p, lpr);
  });
  return last_rc();
}
