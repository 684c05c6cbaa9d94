// Attention whose scores carry a temperature per head and lose a logarithm of the distance,
// over keys in runs of positions: what the paged attention kernels share for it.
//
//   score(i, j) = (q_i . k_j) * scale * temp_h - r1_h ln(1 + r2_h (i - j))
//   key j <= i is visible when floor(i / chunk) = floor(j / chunk)   (chunk 0: always)
//
// A kernel that keeps scores in units of log2 takes the penalty as r1 log2(1 + r2 d), which is
// the same number times log2 e.
#pragma once
#include "common.cuh"

struct IxDistance {
  const float* temp;   // per query head; temp, r1 and r2 are given together or not at all
  const float* r1;
  const float* r2;
  int chunk;           // positions a run spans; 0: no runs
};

// Where a kernel reads queries and writes results: token t of q starts at t * q_ld, of the
// output at t * o_ld (elements); results are multiplied by o_scale before they are rounded.
// What else happens to a (token, head) pair's result where it is normalised and written:
// `sink` (null: none) holds a number per query head whose exponential joins the softmax's
// denominator, a key with that score and no value; `gate` (null: none) holds a number per
// (token, head), row t at t * gate_ld, in the activations' type: the result is multiplied by
// its sigmoid.
struct IxRows {
  long long q_ld, o_ld;
  float o_scale;
  const float* sink;
  const void* gate;
  long long gate_ld;
};

__host__ __device__ __forceinline__ IxDistance ix_no_distance() {
  return IxDistance{nullptr, nullptr, nullptr, 0};
}

// o_scale times the head's gate, where there is one.
template <typename TA>
__device__ __forceinline__ float ix_result_factor(const IxRows& rows, long long token, int head) {
  if (!rows.gate) return rows.o_scale;
  const float z = to_f32(reinterpret_cast<const TA*>(rows.gate)[token * rows.gate_ld + head]);
  return rows.o_scale / (1.0f + expf(-z));
}

// The first key a query at position `pos` can see.
__device__ __forceinline__ int ix_first_key(int pos, int window, int chunk) {
  if (window > 0) return max(0, pos - window + 1);
  if (chunk > 0) return pos / chunk * chunk;
  return 0;
}

__device__ __forceinline__ float ix_log2(float x) {
  float y;
  asm("lg2.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
