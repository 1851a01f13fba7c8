// Ragged batches and activation-type helpers shared by the kernels of the hybrid decoders.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include "sx_api.h"

namespace sx {

// Rows of several sequences, one portion each, packed one after another.
struct RaggedView {
  const int* cu;        // [n + 1] first row of each portion
  const int* pos0;      // [n] position of that row in its sequence (0: the sequence starts here)
  const int* slot;      // [n] state slot
  const int* tok_seq;   // [T] portion of each row
  const int* tok_pos;   // [T] position of each row
  int n;
};
inline RaggedView view(const SxRagged* r) { return RaggedView{r->cu, r->pos0, r->slot, r->tok_seq, r->tok_pos, r->n}; }

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename A> __device__ __forceinline__ A from_f(float x);
template <> __device__ __forceinline__ float from_f<float>(float x) { return x; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}
__device__ __forceinline__ void store4(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, float a, float b, float c, float d) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 v;
  v.x = *reinterpret_cast<unsigned*>(&lo);
  v.y = *reinterpret_cast<unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = v;
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// silu of an activation: 32-bit runs take the accurate forms, 16-bit ones the hardware exponential and reciprocal
template <typename A> __device__ __forceinline__ float silu_act(float x) {
  return sizeof(A) == 4 ? x * sigmoid_f(x) : __fdividef(x, 1.f + __expf(-x));
}
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// NT tokens of one channel of a short causal convolution: y[t] = sum_b w[b] x[t - b]. `u` points at the first token's row;
// tokens in front of it are earlier rows of the portion (s0 of them are there) or come from the ring, which keeps position p
// in entry p % taps; positions before the sequence are zero. w [taps, C], last row for the current token; taps <= MT.
template <typename A, int NT, int MT>
__device__ __forceinline__ void conv_walk(const A* __restrict__ u, long long ld, const float* __restrict__ w, int taps, int C, int ch,
                                          const A* ring, int pos, int s0, int nt, float (&y)[NT]) {
  float x[NT + MT - 1], wb[MT];
#pragma unroll
  for (int b = 0; b < MT; ++b) wb[b] = b < taps ? w[(long long)(taps - 1 - b) * C + ch] : 0.f;
  if (NT > 1 && s0 >= MT - 1 && nt == NT) {     // inside a portion: every row is there
    const A* r = u + ch - (MT - 1) * ld;
    A raw[NT + MT - 1];
#pragma unroll
    for (int i = 0; i < NT + MT - 1; ++i, r += ld) raw[i] = *r;
#pragma unroll
    for (int i = 0; i < NT + MT - 1; ++i) x[i] = to_f(raw[i]);
  } else {
    const int ph = pos % taps;
#pragma unroll
    for (int i = 0; i < NT + MT - 1; ++i) {
      const int t = i - (MT - 1);          // token relative to the first one
      x[i] = 0.f;
      if (t < 0) {
        if (-t < taps) {
          if (s0 + t >= 0) x[i] = to_f(u[(long long)t * ld + ch]);
          else if (pos + t >= 0) x[i] = to_f(ring[(long long)(ph + t >= 0 ? ph + t : ph + t + taps) * C + ch]);
        }
      } else if (t < nt) {
        x[i] = to_f(u[(long long)t * ld + ch]);
      }
    }
  }
#pragma unroll
  for (int t = 0; t < NT; ++t) {
    float a = 0.f;
#pragma unroll
    for (int b = MT - 1; b >= 0; --b) a = fmaf(wb[b], x[t + MT - 1 - b], a);
    y[t] = a;
  }
}

struct ChunkView {
  const int* seq;       // [n_chunks] portion of each chunk
  const int* start;     // [n_chunks] first row of the chunk within its portion
  const int* first;     // [n + 1] first chunk of each portion
  int n_chunks;
};
inline ChunkView chunks(const SxChunks* c) { return ChunkView{c->seq, c->start, c->first, c->n}; }
constexpr int RC = 16;  // rows per chunk

inline int last_rc() { return cudaGetLastError() == cudaSuccess ? 0 : -11; }

}  // namespace sx

#define SX_ACT_DISPATCH(is_f32, ...)              \
  do {                                            \
    if (is_f32) { using A = float; __VA_ARGS__; } \
    else { using A = __nv_bfloat16; __VA_ARGS__; } \
  } while (0)
