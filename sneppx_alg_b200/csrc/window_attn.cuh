// Shared by the kernels of window attention over tokens and averaged blocks.
#pragma once
#include "common.cuh"
#include "ragged.cuh"
#include "sx_api.h"

namespace sx {

struct WinParams {
  SxWinAttnArgs a;
  RaggedView rv;
};

// What a query at `pos` sees: averaged blocks 0 .. blocks - 1, then the tokens first .. pos.
struct WinKeys {
  int blocks, first, tokens;
};
__host__ __device__ __forceinline__ WinKeys win_keys(int pos, int size, int pool) {
  WinKeys k;
  k.first = pos - size + 1 > 0 ? pos - size + 1 : 0;
  k.blocks = k.first / pool;
  k.tokens = pos - k.first + 1;
  return k;
}

// Cache entry of the i-th key of a sequence (blocks first).
__device__ __forceinline__ long long win_entry(const WinParams& P, int seq, const WinKeys& k, int i) {
  const SxWinAttnArgs& p = P.a;
  if (i < k.blocks) return (long long)p.pool_table[(long long)seq * p.pool_ld + i / p.block_size] * p.block_size + i % p.block_size;
  const int j = k.first + i - k.blocks;
  return (long long)p.block_table[(long long)seq * p.table_ld + j / p.block_size - p.block_base[seq]] * p.block_size + j % p.block_size;
}

// Pair e of head h of an output row: turned back by the row's angle, gated and stored.
template <typename A>
__device__ __forceinline__ void win_store(const WinParams& P, long long t, int h, int e, int2 at, float a, float b) {
  const SxWinAttnArgs& p = P.a;
  const float2 cs = reinterpret_cast<const float2*>(p.turn)[t * (p.dv / 2) + e];
  const A* gate = reinterpret_cast<const A*>(p.gate) + t * p.gate_ld + (long long)h * p.dv;
  A* y = reinterpret_cast<A*>(p.y) + t * p.y_ld + (long long)h * p.dv;
  y[at.x] = from_f<A>((a * cs.x + b * cs.y) * sigmoid_f(to_f(gate[at.x])));
  y[at.y] = from_f<A>((b * cs.x - a * cs.y) * sigmoid_f(to_f(gate[at.y])));
}

}  // namespace sx
