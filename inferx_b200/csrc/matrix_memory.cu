// A matrix memory with exponential gates and a normaliser, per head and request.
//
//   log gates      i_t = cap tanh((W_i h + b_i) / cap),  f_t = logsigmoid(cap tanh((W_f h + b_f) / cap))
//   running max    m_t = max(f_t + m_(t-1), i_t), m = 0 before a sequence's first token
//   keep, put      exp(f_t + m_(t-1) - m_t),  exp(i_t - m_t);  floor = exp(-m_t)
//   memory         S_t = keep S_(t-1) + put k_t v_t^T,  n_t = keep n_(t-1) + put k_t
//   read-out       num_t = S_t^T q_t,  nq_t = n_t . q_t
//
// The head's output num / (max(|nq|, floor) + eps) is formed with the norm and the gate that
// follow: in these kernels where a block has the whole head (MmFinish), else by
// ix_head_norm_gate.  S [slots, H, K, V], n [slots, H, K] and m [slots, H] are fp32 state per
// request.  Three kernels make the gates: one for steps of single tokens, which also takes the
// dot products; a scan over each sequence otherwise (the two numbers of a token combine
// associatively: the sum of the f's and the largest i carried to the end).  The memory is
// walked by one of three forms: single tokens (the memory streams through the chip once),
// token by token with the memory in registers (any sizes and types), and in chunks
// (matrix_memory_chunks.cu).
#include "matrix_memory.cuh"

__device__ __forceinline__ float mm_cap(float z, float cap) { return cap * tanhf(z / cap); }
// logsigmoid(z) = min(z, 0) - log(1 + exp(-|z|))
__device__ __forceinline__ float mm_log_sigmoid(float z) {
  return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// ---------------------------------------------------------------------------
// Steps of single tokens: one warp per (token, head) forms both dot products and moves the
// running maximum on.  x [T, W] and w [2 H, W] (input gates' rows, then forget gates') of one
// type; gates [4, H, T]: keep, put, floor and
// the logarithm of keep.
// ---------------------------------------------------------------------------
#define MG_WARPS 4

template <typename TA, bool VEC>
__global__ void __launch_bounds__(MG_WARPS * 32)
mm_gates_single_kernel(const TA* __restrict__ x, const TA* __restrict__ w,
                       const float* __restrict__ bias, float cap, float* __restrict__ m_state,
                       const int* __restrict__ state_slot, float* __restrict__ gates, int T, int W,
                       int H) {
  IX_PDL_WAIT();
  const int lane = threadIdx.x & 31;
  const int pair = blockIdx.x * MG_WARPS + (threadIdx.x >> 5);
  if (pair >= T * H) return;
  const int t = pair / H, h = pair - t * H;
  const TA* xr = x + (size_t)t * W;
  const TA* wi = w + (size_t)h * W;
  const TA* wf = w + (size_t)(H + h) * W;
  float zi = 0.f, zf = 0.f;
  if (VEC) {                        // bf16, W a multiple of 8: 16-byte accesses
#pragma unroll 4
    for (int c = lane * 8; c < W; c += 256) {
      const uint4 a = *reinterpret_cast<const uint4*>(xr + c);
      const uint4 b = *reinterpret_cast<const uint4*>(wi + c);
      const uint4 d = *reinterpret_cast<const uint4*>(wf + c);
      const __nv_bfloat162* pa = reinterpret_cast<const __nv_bfloat162*>(&a);
      const __nv_bfloat162* pb = reinterpret_cast<const __nv_bfloat162*>(&b);
      const __nv_bfloat162* pd = reinterpret_cast<const __nv_bfloat162*>(&d);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 fa = __bfloat1622float2(pa[e]), fb = __bfloat1622float2(pb[e]),
                     fd = __bfloat1622float2(pd[e]);
        zi = fmaf(fa.x, fb.x, zi); zi = fmaf(fa.y, fb.y, zi);
        zf = fmaf(fa.x, fd.x, zf); zf = fmaf(fa.y, fd.y, zf);
      }
    }
  } else {
    for (int c = lane; c < W; c += 32) {
      const float v = to_f32(xr[c]);
      zi = fmaf(v, to_f32(wi[c]), zi);
      zf = fmaf(v, to_f32(wf[c]), zf);
    }
  }
  zi = warp_sum(zi);
  zf = warp_sum(zf);
  if (lane == 0) {
    const float i = mm_cap(zi + bias[h], cap), f = mm_log_sigmoid(mm_cap(zf + bias[H + h], cap));
    float* mp = m_state + (size_t)state_slot[t] * H + h;     // token t is sequence t
    const float before = *mp;
    const float m = fmaxf(f + before, i);
    *mp = m;
    const size_t at = (size_t)h * T + t, plane = (size_t)T * H;
    gates[at] = expf(f + before - m);
    gates[plane + at] = expf(i - m);
    gates[2 * plane + at] = expf(-m);
    gates[3 * plane + at] = f + before - m;
  }
}

IX_API int ix_mm_gates_single(const void* x, const void* w, int dtype, const float* bias,
                              float cap, float* m_state, const int* state_slot, float* gates,
                              int T, int W, int H, cudaStream_t stream) {
  if (T <= 0) return IX_OK;
  if (W <= 0 || H <= 0 || !(cap > 0.f)) return IX_ERR_SIZE;
  const long long pairs = (long long)T * H;
  const unsigned blocks = (unsigned)((pairs + MG_WARPS - 1) / MG_WARPS);
  const bool vec = dtype == IX_BF16 && W % 8 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0;
  if (vec)
    ix_launch(mm_gates_single_kernel<bf16, true>, dim3(blocks), dim3(MG_WARPS * 32), 0, stream,
              (const bf16*)x, (const bf16*)w, bias, cap, m_state, state_slot, gates, T, W, H);
  else
    IX_DISPATCH_DTYPE(dtype, TA,
                      ix_launch(mm_gates_single_kernel<TA, false>, dim3(blocks),
                                dim3(MG_WARPS * 32), 0, stream, (const TA*)x, (const TA*)w, bias,
                                cap, m_state, state_slot, gates, T, W, H));
  return ix_launch_status();
}

// ---------------------------------------------------------------------------
// Any step: z fp32 [2 H, T] holds the dot products; one block per (head, sequence) walks the
// sequence in tiles of a token per thread.  A span of tokens is the pair (F, M): m at its
// end is max(m before it + F, M); spans join as (F1 + F2, max(M1 + F2, M2)).  keep uses the
// m of the token before as that token's own thread formed it.
// ---------------------------------------------------------------------------
#define MS_THREADS 1024

__global__ void __launch_bounds__(MS_THREADS)
mm_gates_scan_kernel(const float* __restrict__ z, const float* __restrict__ bias, float cap,
                     float* __restrict__ m_state, const int* __restrict__ state_slot,
                     const int* __restrict__ cu_q, float* __restrict__ gates, int T, int H) {
  __shared__ float wF[MS_THREADS / 32], wM[MS_THREADS / 32], last[MS_THREADS / 32];
  IX_PDL_WAIT();
  const int h = blockIdx.x, s = blockIdx.y;
  const int begin = cu_q[s], end = cu_q[s + 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* mp = m_state + (size_t)state_slot[s] * H + h;
  float carry = *mp;
  const float bi = bias[h], bf = bias[H + h];
  const size_t plane = (size_t)T * H;
  for (int t0 = begin; t0 < end; t0 += MS_THREADS) {
    const int t = t0 + threadIdx.x;
    const bool ok = t < end;
    float i = -INFINITY, f = 0.f;          // past the end: a span that changes nothing
    if (ok) {
      i = mm_cap(z[(size_t)h * T + t] + bi, cap);
      f = mm_log_sigmoid(mm_cap(z[(size_t)(H + h) * T + t] + bf, cap));
    }
    float F = f, M = i;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pF = __shfl_up_sync(0xffffffffu, F, o), pM = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) {
        M = fmaxf(pM + F, M);
        F = pF + F;
      }
    }
    if (lane == 31) {
      wF[warp] = F;
      wM[warp] = M;
    }
    __syncthreads();
    float m0 = carry;                       // m before this warp's first token
    for (int w = 0; w < warp; ++w) m0 = fmaxf(m0 + wF[w], wM[w]);
    const float m = fmaxf(m0 + F, M);
    if (lane == 31) last[warp] = m;
    __syncthreads();
    float before = __shfl_up_sync(0xffffffffu, m, 1);
    if (lane == 0) before = warp == 0 ? carry : last[warp - 1];
    if (ok) {
      const size_t at = (size_t)h * T + t;
      gates[at] = expf(f + before - m);
      gates[plane + at] = expf(i - m);
      gates[2 * plane + at] = expf(-m);
      gates[3 * plane + at] = f + before - m;
    }
    carry = last[MS_THREADS / 32 - 1];
    __syncthreads();
  }
  if (threadIdx.x == 0 && end > begin) *mp = carry;
}

IX_API int ix_mm_gates_scan(const float* z, const float* bias, float cap, float* m_state,
                            const int* state_slot, const int* cu_q, float* gates, int T, int S,
                            int H, cudaStream_t stream) {
  if (T <= 0 || S <= 0) return IX_OK;
  if (H <= 0 || S > 65535 || !(cap > 0.f)) return IX_ERR_SIZE;
  ix_launch(mm_gates_scan_kernel, dim3(H, S), dim3(MS_THREADS), 0, stream, z, bias, cap, m_state,
            state_slot, cu_q, gates, T, H);
  return ix_launch_status();
}

// ---------------------------------------------------------------------------
// Single tokens: sequence s is token s.  A block owns MD_COLS value columns of one (sequence,
// head): every row of its part of the memory is read, moved on, multiplied into the outputs
// and written once; eight warps split the rows.  The block of the first columns keeps the
// normaliser.
// ---------------------------------------------------------------------------
#define MD_WARPS 8
#define MD_COLS 128
#define MD_ROWS 8       // rows a warp has in flight

// With `fin.gain` (V at most MD_COLS: the block has the head's whole output) the block divides
// by the normaliser, norms, gates and writes the head's row of the activations itself.
template <typename TA, bool VEC>
__global__ void __launch_bounds__(MD_WARPS * 32)
mm_single_kernel(const TA* __restrict__ q, long long ldq, const TA* __restrict__ k, long long ldk,
                 const TA* __restrict__ v, long long ldv, const float* __restrict__ gates,
                 float* __restrict__ S, float* __restrict__ N, const int* __restrict__ state_slot,
                 float* __restrict__ num, float* __restrict__ nq, int T, int H, int K, int V,
                 float q_scale, MmFinish fin) {
  extern __shared__ __align__(16) float sm[];
  float* q_s = sm;             // [K]
  float* k_s = sm + K;         // [K], times put
  float* part = sm + ((2 * K + 3) & ~3);    // [MD_WARPS][MD_COLS]
  __shared__ float scratch[32];
  IX_PDL_WAIT();
  const int t = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * MD_COLS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t at = (size_t)t * H + h, plane = (size_t)T * H;
  const size_t gate_at = (size_t)h * T + t;
  const float keep = gates[gate_at], put = gates[plane + gate_at];
  const size_t slot_head = (size_t)state_slot[t] * H + h;
  for (int i = tid; i < K; i += MD_WARPS * 32) {
    q_s[i] = to_f32(q[t * ldq + (size_t)h * K + i]) * q_scale;
    k_s[i] = to_f32(k[t * ldk + (size_t)h * K + i]) * put;
  }
  __syncthreads();
  float* st = S + slot_head * K * V;
  const TA* vr = v + t * ldv + (size_t)h * V;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  if (VEC) {
    const int c = v0 + lane * 4;
    if (c < V) {
      float vv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) vv[e] = to_f32(vr[c + e]);
      for (int r0 = warp; r0 < K; r0 += MD_WARPS * MD_ROWS) {
        float4 x[MD_ROWS];
#pragma unroll
        for (int j = 0; j < MD_ROWS; ++j) {
          const int r = r0 + j * MD_WARPS;
          if (r < K) x[j] = *reinterpret_cast<const float4*>(st + (size_t)r * V + c);
        }
#pragma unroll
        for (int j = 0; j < MD_ROWS; ++j) {
          const int r = r0 + j * MD_WARPS;
          if (r >= K) break;
          const float kk = k_s[r], qq = q_s[r];
          x[j].x = fmaf(keep, x[j].x, kk * vv[0]);
          x[j].y = fmaf(keep, x[j].y, kk * vv[1]);
          x[j].z = fmaf(keep, x[j].z, kk * vv[2]);
          x[j].w = fmaf(keep, x[j].w, kk * vv[3]);
          acc[0] = fmaf(x[j].x, qq, acc[0]);
          acc[1] = fmaf(x[j].y, qq, acc[1]);
          acc[2] = fmaf(x[j].z, qq, acc[2]);
          acc[3] = fmaf(x[j].w, qq, acc[3]);
          *reinterpret_cast<float4*>(st + (size_t)r * V + c) = x[j];
        }
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) part[warp * MD_COLS + lane * 4 + e] = acc[e];
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = v0 + e * 32 + lane;
      if (c < V) {
        const float vv = to_f32(vr[c]);
        for (int r = warp; r < K; r += MD_WARPS) {
          const float x = fmaf(keep, st[(size_t)r * V + c], k_s[r] * vv);
          acc[e] = fmaf(x, q_s[r], acc[e]);
          st[(size_t)r * V + c] = x;
        }
      }
      part[warp * MD_COLS + e * 32 + lane] = acc[e];
    }
  }
  __syncthreads();
  float total = 0.f;                 // of column tid (MD_COLS threads have one)
  if (tid < MD_COLS && v0 + tid < V) {
#pragma unroll
    for (int w = 0; w < MD_WARPS; ++w) total += part[w * MD_COLS + tid];
    if (!fin.gain) num[at * V + v0 + tid] = total;
  }
  if (blockIdx.x == 0) {
    float* nr = N + slot_head * K;
    float a = 0.f;
    for (int i = tid; i < K; i += MD_WARPS * 32) {
      const float x = fmaf(keep, nr[i], k_s[i]);
      a = fmaf(x, q_s[i], a);
      nr[i] = x;
    }
    a = block_sum(a, scratch);
    if (fin.gain) {
      const float y = total / (fmaxf(fabsf(a), gates[2 * plane + gate_at]) + fin.den_eps);
      const float ss = block_sum(y * y, scratch);     // 0 beyond V
      if (tid < V) {
        const size_t c = (size_t)h * V + tid;
        const float z = to_f32(reinterpret_cast<const TA*>(fin.gate)[(size_t)t * fin.gate_ld + c]);
        reinterpret_cast<TA*>(fin.out)[(size_t)t * H * V + c] =
            from_f32<TA>(y / sqrtf(ss / (float)V + fin.eps) * fin.gain[c] / (1.0f + expf(-z)));
      }
    } else if (tid == 0) {
      nq[at] = a;
    }
  }
}

// q, k [T, H K] and v [T, H V] are views with row pitches; sequences 0 .. singles - 1 bring one
// token each (token s of the step).  gates [4, H, T] as the gate kernels leave them.  num fp32
// [T, H, V], nq fp32 [T, H]; or, with `gain`, the finished rows in `out` (see MmFinish).
IX_API int ix_mm_single(const void* q, long long ldq, const void* k, long long ldk,
                        const void* v, long long ldv, int dtype, const float* gates, float* S,
                        float* N, const int* state_slot, float* num, float* nq, int T,
                        int singles, int H, int K, int V, float q_scale, const float* gain,
                        const void* gate, long long gate_ld, float eps, float den_eps, void* out,
                        cudaStream_t stream) {
  if (singles <= 0) return IX_OK;
  if (gain && (V > MD_COLS || !gate || !out)) return IX_ERR_UNSUPPORTED;
  const MmFinish fin = {gain, gate, gate_ld, eps, den_eps, out};
  if (H <= 0 || K <= 0 || V <= 0 || H > 65535 || singles > 65535 || singles > T)
    return IX_ERR_SIZE;
  const size_t smem = ((size_t)((2 * K + 3) & ~3) + MD_WARPS * MD_COLS) * sizeof(float);
  if (smem > 48 * 1024) return IX_ERR_SMEM;
  const bool vec = V % 4 == 0 && ((uintptr_t)S & 15) == 0;
  const dim3 grid((V + MD_COLS - 1) / MD_COLS, H, singles);
  IX_DISPATCH_DTYPE(dtype, TA, {
    auto kern = vec ? mm_single_kernel<TA, true> : mm_single_kernel<TA, false>;
    ix_launch(kern, grid, dim3(MD_WARPS * 32), smem, stream, (const TA*)q, ldq, (const TA*)k, ldk,
              (const TA*)v, ldv, gates, S, N, state_slot, num, nq, T, H, K, V, q_scale,
              fin);
  });
  return ix_launch_status();
}

// ---------------------------------------------------------------------------
// Token by token: grid (ceil(V / 32) + 1, heads, sequences); a block is 32 value columns times
// KS slices of the key entries (a warp a slice); a thread keeps its KPT entries of one column
// in registers from the sequence's first token of the step to its last.  The last block of a
// head keeps the normaliser as one more column whose value is always one.
// ---------------------------------------------------------------------------
#define MW_COLS 32
#define MW_CHUNK 16

template <typename TA, int KPT>
__global__ void __launch_bounds__(MW_COLS * 8)
mm_walk_kernel(const TA* __restrict__ q, long long ldq, const TA* __restrict__ k, long long ldk,
               const TA* __restrict__ v, long long ldv, const float* __restrict__ gates,
               float* __restrict__ S, float* __restrict__ N, const int* __restrict__ cu_q,
               const int* __restrict__ state_slot, float* __restrict__ num,
               float* __restrict__ nq, int T, int H, int K, int V, int KS, int s0,
               float q_scale) {
  extern __shared__ __align__(16) float sm[];
  float* q_s = sm;                          // [MW_CHUNK][K]
  float* k_s = q_s + MW_CHUNK * K;          // [MW_CHUNK][K], times put
  float* v_s = k_s + MW_CHUNK * K;          // [MW_CHUNK][MW_COLS]
  float* part = v_s + MW_CHUNK * MW_COLS;   // [KS][MW_CHUNK][MW_COLS]
  __shared__ float keep_s[MW_CHUNK];
  IX_PDL_WAIT();
  const int lane = threadIdx.x & 31, ks = threadIdx.x >> 5;
  const bool norm = blockIdx.x == gridDim.x - 1;
  const int v0 = blockIdx.x * MW_COLS, h = blockIdx.y, s = s0 + blockIdx.z;
  const int col = norm ? lane : v0 + lane;
  const bool col_ok = norm ? lane == 0 : col < V;
  const int begin = cu_q[s], end = cu_q[s + 1];
  const size_t slot_head = (size_t)state_slot[s] * H + h;
  float* st = norm ? N + slot_head * K : S + slot_head * K * V;
  const int pitch = norm ? 1 : V;
  const int kk0 = ks * KPT;
  const size_t plane = (size_t)T * H;
  float x[KPT];
#pragma unroll
  for (int i = 0; i < KPT; ++i)
    x[i] = (kk0 + i < K && col_ok) ? st[(size_t)(kk0 + i) * pitch + col] : 0.f;
  for (int t0 = begin; t0 < end; t0 += MW_CHUNK) {
    const int n = min(MW_CHUNK, end - t0);
    for (int i = threadIdx.x; i < n * K; i += blockDim.x) {
      const int c = i / K, kk = i - c * K;
      const size_t t = (size_t)(t0 + c);
      q_s[i] = to_f32(q[t * ldq + (size_t)h * K + kk]) * q_scale;
      k_s[i] = to_f32(k[t * ldk + (size_t)h * K + kk]) * gates[plane + (size_t)h * T + t];
    }
    for (int i = threadIdx.x; i < n * MW_COLS; i += blockDim.x) {
      const int c = i / MW_COLS, j = i % MW_COLS;
      v_s[i] = norm ? 1.f
                    : (v0 + j < V ? to_f32(v[(size_t)(t0 + c) * ldv + (size_t)h * V + v0 + j])
                                  : 0.f);
    }
    if (threadIdx.x < n) keep_s[threadIdx.x] = gates[(size_t)h * T + t0 + threadIdx.x];
    __syncthreads();
    for (int c = 0; c < n; ++c) {
      const float vj = v_s[c * MW_COLS + lane], keep = keep_s[c];
      const float* kc = k_s + c * K + kk0;
      const float* qc = q_s + c * K + kk0;
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        if (kk0 + i < K) {
          x[i] = fmaf(keep, x[i], kc[i] * vj);
          acc = fmaf(x[i], qc[i], acc);
        }
      }
      part[(ks * MW_CHUNK + c) * MW_COLS + lane] = acc;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * MW_COLS; i += blockDim.x) {
      const int c = i / MW_COLS, j = i % MW_COLS;
      if (norm ? j == 0 : v0 + j < V) {
        float total = 0.f;
        for (int w = 0; w < KS; ++w) total += part[(w * MW_CHUNK + c) * MW_COLS + j];
        const size_t at = (size_t)(t0 + c) * H + h;
        if (norm) nq[at] = total;
        else num[at * V + v0 + j] = total;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < KPT; ++i)
    if (kk0 + i < K && col_ok) st[(size_t)(kk0 + i) * pitch + col] = x[i];
}

IX_API int ix_mm_max_dim() { return 8 * 64; }

// Sequences s0 .. S - 1 of the step, whatever they bring.
IX_API int ix_mm_walk(const void* q, long long ldq, const void* k, long long ldk, const void* v,
                      long long ldv, int dtype, const float* gates, float* S_state, float* N,
                      const int* cu_q, const int* state_slot, float* num, float* nq, int T,
                      int S, int s0, int H, int K, int V, float q_scale, cudaStream_t stream) {
  if (S - s0 <= 0) return IX_OK;
  if (s0 < 0 || H <= 0 || K <= 0 || V <= 0 || K > 8 * 64 || H > 65535 || S > 65535)
    return IX_ERR_SIZE;
  const int KS = K > 32 ? 8 : (K > 8 ? 4 : 1);
  const int kpt = (K + KS - 1) / KS;
  const size_t smem = ((size_t)2 * MW_CHUNK * K + MW_CHUNK * MW_COLS +
                       (size_t)KS * MW_CHUNK * MW_COLS) * sizeof(float);
  if (smem > 200 * 1024) return IX_ERR_SMEM;
  const dim3 grid((V + MW_COLS - 1) / MW_COLS + 1, H, S - s0), block(MW_COLS * KS);
#define MW_GO(KPT)                                                                             \
  IX_DISPATCH_DTYPE(dtype, TA, {                                                               \
    auto kern = mm_walk_kernel<TA, KPT>;                                                       \
    if (smem > 48 * 1024)                                                                      \
      cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
    ix_launch(kern, grid, block, smem, stream, (const TA*)q, ldq, (const TA*)k, ldk,           \
              (const TA*)v, ldv, gates, S_state, N, cu_q, state_slot, num, nq, T, H, K, V, KS, \
              s0, q_scale);                                                                    \
  })
  if (kpt <= 8) MW_GO(8);
  else if (kpt <= 16) MW_GO(16);
  else if (kpt <= 32) MW_GO(32);
  else MW_GO(64);
#undef MW_GO
  return ix_launch_status();
}
