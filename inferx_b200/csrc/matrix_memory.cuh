// What the kernels of the matrix memory share.
#pragma once
#include "common.cuh"

// A head's row on its way out: y = num / (max(|nq|, floor) + den_eps), then y / sqrt(mean(y^2) +
// eps) * gain * sigmoid(gate).  gain [H V] fp32 (null: not here); gate: row t at t * gate_ld, H V
// entries in the activations' type, like out [T, H V].
struct MmFinish {
  const float* gain;
  const void* gate;
  long long gate_ld;
  float eps, den_eps;
  void* out;
};
