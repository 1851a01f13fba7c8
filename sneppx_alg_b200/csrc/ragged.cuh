// Ragged batches and activation-type helpers shared by the kernels of the hybrid decoders.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include "sx_api.h"

namespace sx {

constexpr int QK_PAIRS = 4;   // a lane holds up to this many pairs of a query / key head: head sizes up to 256

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
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

inline int last_rc() { return cudaGetLastError() == cudaSuccess ? 0 : -11; }

}  // namespace sx

#define SX_ACT_DISPATCH(is_f32, ...)              \
  do {                                            \
    if (is_f32) { using A = float; __VA_ARGS__; } \
    else { using A = __nv_bfloat16; __VA_ARGS__; } \
  } while (0)
