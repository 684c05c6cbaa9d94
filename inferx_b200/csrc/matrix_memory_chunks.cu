// The matrix memory of matrix_memory.cu over portions of prompts, in chunks on the tensor
// cores (bfloat16 q, k, v).
//
// Inside a chunk of 64 tokens, with G_t the sum of the log keeps up to and with token t:
//
//   num_t = exp(G_t) S_start^T q_t + sum_(s <= t) exp(G_t - G_s) put_s (q_t . k_s) v_s
//   nq_t  = exp(G_t) n_start . q_t + sum_(s <= t) exp(G_t - G_s) put_s (q_t . k_s)
//   S_end = exp(G_end) S_start + sum_s exp(G_end - G_s) put_s k_s v_s^T      (n likewise)
//
// Three passes, each over all chunks of all sequences at once or over all entries of the
// memory at once:
//   own    every chunk's own sum into S_end and n_end, to scratch            (tensor cores)
//   join   per entry of the memory, along a sequence's chunks: the scratch entry becomes
//          the chunk's start state, split into two bfloat16 terms; the state moves on
//   out    num and nq of every token                                         (tensor cores)
// The memory, its sums and the gates are fp32; where fp32 numbers enter a tensor-core product
// (the weighted keys, the weighted scores, the start state) they enter as two bfloat16 terms
// each (16 bits) into the same fp32 accumulator, and q, k and v as they are.  A chunk's scratch
// number is tokens before the sequence / 64 + the sequence's number + the chunk's: no two meet.
#include "matrix_memory.cuh"

#define MC_L 64               // tokens a chunk
#define MC_THREADS 128
#define MC_WARPS 4

__device__ __forceinline__ unsigned mc_smem(const void* p) {
  return (unsigned)__cvta_generic_to_shared(p);
}
__device__ __forceinline__ void mc_ldm4(unsigned* r, unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mc_ldm4t(unsigned* r, unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mc_mma(float* c, const unsigned* a, unsigned b0, unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
      "{%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned mc_pack(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const unsigned*>(&v);
}
// what a pair loses in mc_pack, packed
__device__ __forceinline__ unsigned mc_pack_rest(float a, float b, unsigned hi) {
  const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&hi);
  return mc_pack(a - __low2float(h), b - __high2float(h));
}

// 16 or 8 bytes to shared memory without registers in between; `bytes` of them are read, the
// rest is zero
__device__ __forceinline__ void mc_async16(void* dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mc_smem(dst)), "l"(src),
               "r"(bytes) : "memory");
}
__device__ __forceinline__ void mc_async8(void* dst, const void* src, int bytes) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(mc_smem(dst)), "l"(src),
               "r"(bytes) : "memory");
}
__device__ __forceinline__ void mc_async_wait() {
  asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
}

// `rows` of MC_L rows (the rest zero) of `cols` entries into shared rows of `pitch` entries,
// columns cols .. padded zero.  vec: rows start on 16-byte marks and cols is a multiple of 8; the
// copies are then asynchronous (mc_async_wait).
__device__ __forceinline__ void mc_load(bf16* dst, int pitch, const bf16* src, long long ld,
                                        int rows, int cols, int padded, bool vec) {
  if (vec) {
    const int per = padded >> 3;
    for (int i = threadIdx.x; i < MC_L * per; i += MC_THREADS) {
      const int r = i / per, c = (i - r * per) * 8;
      const bool ok = r < rows && c < cols;
      mc_async16(dst + r * pitch + c, ok ? src + (size_t)r * ld + c : src, ok ? 16 : 0);
    }
  } else {
    for (int i = threadIdx.x; i < MC_L * padded; i += MC_THREADS) {
      const int r = i / padded, c = i - r * padded;
      dst[r * pitch + c] = (r < rows && c < cols) ? src[(size_t)r * ld + c] : __float2bfloat16_rn(0.f);
    }
  }
}

// G of the chunk's tokens and put by one warp; tokens past the end: G of the last, put 0.
__device__ __forceinline__ void mc_gates(float* G, float* put, const float* gates, size_t plane,
                                         size_t first, int n) {
  const int lane = threadIdx.x & 31;
  float carry = 0.f;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = half * 32 + lane;
    float g = t < n ? gates[3 * plane + first + t] : 0.f;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float p = __shfl_up_sync(0xffffffffu, g, o);
      if (lane >= o) g += p;
    }
    g += carry;
    carry = __shfl_sync(0xffffffffu, g, 31);
    G[t] = g;
    put[t] = t < n ? gates[plane + first + t] : 0.f;
  }
}

struct McWhere {           // one block's chunk
  int t0, n, entry;        // first token of the step, tokens, scratch number
};
__device__ __forceinline__ McWhere mc_where(const int* cu_q, int s, int s0, int chunk) {
  const int begin = cu_q[s], end = cu_q[s + 1], base = cu_q[s0];
  McWhere w;
  w.t0 = begin + chunk * MC_L;
  w.n = min(MC_L, end - w.t0);
  w.entry = (begin - base) / MC_L + (s - s0) + chunk;
  return w;
}

// ---------------------------------------------------------------------------
// own: grid (V tiles, chunks, heads * sequences)
// ---------------------------------------------------------------------------
template <int VT>
__global__ void __launch_bounds__(MC_THREADS)
mm_chunk_own_kernel(const bf16* __restrict__ k, long long ldk, const bf16* __restrict__ v,
                    long long ldv, const float* __restrict__ gates, const int* __restrict__ cu_q,
                    float* __restrict__ scr_s, float* __restrict__ scr_n, float* __restrict__ scr_p,
                    int T, int H, int K, int V, int s0, int vec_k, int vec_v) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ float G[MC_L], put[MC_L];
  const int Kp = (K + 15) & ~15, Vp = (V + 7) & ~7;
  const int pk = Kp + 8, pv = VT + 8;
  bf16* k_hi = reinterpret_cast<bf16*>(smem_raw);       // [MC_L][pk]
  bf16* k_lo = k_hi + MC_L * pk;
  bf16* v_s = k_lo + MC_L * pk;                         // [MC_L][pv]
  const int h = blockIdx.z % H, s = s0 + blockIdx.z / H, v0 = blockIdx.x * VT;
  const McWhere at = mc_where(cu_q, s, s0, blockIdx.y);
  if (at.n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t plane = (size_t)T * H;
  mc_load(k_hi, pk, k + (size_t)at.t0 * ldk + (size_t)h * K, ldk, at.n, K, Kp, vec_k);
  mc_load(v_s, pv, v + (size_t)at.t0 * ldv + (size_t)h * V + v0, ldv, at.n, min(VT, V - v0), VT,
          vec_v);
  if (warp == 0) mc_gates(G, put, gates, plane, (size_t)h * T + at.t0, at.n);
  mc_async_wait();
  __syncthreads();
  const float g_end = G[MC_L - 1];
  // the keys times their weight at the chunk's end, in two terms
  for (int i = tid; i < MC_L * (Kp >> 1); i += MC_THREADS) {
    const int t = i / (Kp >> 1), c = (i - t * (Kp >> 1)) * 2;
    const float w = expf(g_end - G[t]) * put[t];
    const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(k_hi + t * pk + c);
    const float a = __low2float(x) * w, b = __high2float(x) * w;
    const unsigned hi = mc_pack(a, b);
    *reinterpret_cast<unsigned*>(k_hi + t * pk + c) = hi;
    *reinterpret_cast<unsigned*>(k_lo + t * pk + c) = mc_pack_rest(a, b, hi);
  }
  __syncthreads();
  const size_t cell = (size_t)at.entry * H + h;
  if (blockIdx.x == 0) {
    for (int c = tid; c < K; c += MC_THREADS) {
      float sum = 0.f;
      for (int t = 0; t < at.n; ++t)
        sum += __bfloat162float(k_hi[t * pk + c]) + __bfloat162float(k_lo[t * pk + c]);
      scr_n[cell * K + c] = sum;
    }
    if (tid == 0) scr_p[cell] = expf(g_end);
  }
  float* out = scr_s + cell * K * Vp;
  for (int mt = warp; mt < Kp >> 4; mt += MC_WARPS) {
    float acc[VT / 8][4];
#pragma unroll
    for (int j = 0; j < VT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    const int steps = (at.n + 15) >> 4;
    for (int kk = 0; kk < steps; ++kk) {
      unsigned a[4], al[4];
      const int row = kk * 16 + (lane & 7) + ((lane >> 4) & 1) * 8;
      const int col = mt * 16 + ((lane >> 3) & 1) * 8;
      mc_ldm4t(a, mc_smem(k_hi + row * pk + col));
      mc_ldm4t(al, mc_smem(k_lo + row * pk + col));
      const int brow = kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int j = 0; j < VT / 8; j += 2) {
        unsigned b[4];
        mc_ldm4t(b, mc_smem(v_s + brow * pv + j * 8 + ((lane >> 4) & 1) * 8));
        mc_mma(acc[j], a, b[0], b[1]);
        mc_mma(acc[j + 1], a, b[2], b[3]);
        mc_mma(acc[j], al, b[0], b[1]);
        mc_mma(acc[j + 1], al, b[2], b[3]);
      }
    }
    const int g = lane >> 2, t2 = (lane & 3) * 2;
#pragma unroll
    for (int j = 0; j < VT / 8; ++j) {
      const int c = v0 + j * 8 + t2;
      if (c >= Vp) continue;
      const int r = mt * 16 + g;
      if (r < K) *reinterpret_cast<float2*>(out + (size_t)r * Vp + c) = make_float2(acc[j][0], acc[j][1]);
      if (r + 8 < K)
        *reinterpret_cast<float2*>(out + (size_t)(r + 8) * Vp + c) = make_float2(acc[j][2], acc[j][3]);
    }
  }
}

// ---------------------------------------------------------------------------
// join: grid (groups of entries, heads, sequences); a thread owns four neighbouring value
// columns of one row of the memory (or one entry of the normaliser) along the sequence.
// A scratch cell of four fp32 numbers becomes four high terms and four low terms.
// ---------------------------------------------------------------------------
#define MJ_THREADS 128
#define MJ_AHEAD 8

__global__ void __launch_bounds__(MJ_THREADS)
mm_chunk_join_kernel(float* __restrict__ scr_s, float* __restrict__ scr_n,
                     const float* __restrict__ scr_p, float* __restrict__ S,
                     float* __restrict__ N, const int* __restrict__ cu_q,
                     const int* __restrict__ state_slot, int H, int K, int V, int s0) {
  const int h = blockIdx.y, s = s0 + blockIdx.z;
  const McWhere first = mc_where(cu_q, s, s0, 0);
  const int n = cu_q[s + 1] - cu_q[s];
  if (n <= 0) return;
  const int chunks = (n + MC_L - 1) / MC_L;
  const int Vp = (V + 7) & ~7, quads = K * (Vp >> 2);
  const int i = blockIdx.x * MJ_THREADS + threadIdx.x;
  const size_t slot_head = (size_t)state_slot[s] * H + h;
  const size_t cell0 = (size_t)first.entry * H + h;     // chunk c: cell0 + c H
  if (i < quads) {
    const int r = i / (Vp >> 2), c = (i - r * (Vp >> 2)) * 4;
    float* st = S + (slot_head * K + r) * V + c;
    float x[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = c + e < V ? st[e] : 0.f;
    for (int c0 = 0; c0 < chunks; c0 += MJ_AHEAD) {
      float4 own[MJ_AHEAD];
      float p[MJ_AHEAD];
#pragma unroll
      for (int j = 0; j < MJ_AHEAD; ++j)
        if (c0 + j < chunks) {
          const size_t cell = cell0 + (size_t)(c0 + j) * H;
          own[j] = reinterpret_cast<const float4*>(scr_s + cell * K * Vp)[i];
          p[j] = scr_p[cell];
        }
#pragma unroll
      for (int j = 0; j < MJ_AHEAD; ++j)
        if (c0 + j < chunks) {
          const size_t cell = cell0 + (size_t)(c0 + j) * H;
          uint4 w;
          w.x = mc_pack(x[0], x[1]);
          w.y = mc_pack(x[2], x[3]);
          w.z = mc_pack_rest(x[0], x[1], w.x);
          w.w = mc_pack_rest(x[2], x[3], w.y);
          reinterpret_cast<uint4*>(scr_s + cell * K * Vp)[i] = w;
          x[0] = fmaf(p[j], x[0], own[j].x);
          x[1] = fmaf(p[j], x[1], own[j].y);
          x[2] = fmaf(p[j], x[2], own[j].z);
          x[3] = fmaf(p[j], x[3], own[j].w);
        }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (c + e < V) st[e] = x[e];
  } else if (i < quads + K) {
    const int r = i - quads;
    float* st = N + slot_head * K + r;
    float x = *st;
    for (int c = 0; c < chunks; ++c) {
      const size_t cell = cell0 + (size_t)c * H;
      const float own = scr_n[cell * K + r], p = scr_p[cell];
      scr_n[cell * K + r] = x;
      x = fmaf(p, x, own);
    }
    *st = x;
  }
}

// ---------------------------------------------------------------------------
// out: grid (V tiles, chunks, heads * sequences); warp w owns the chunk's tokens 16 w .. 16 w + 15
// ---------------------------------------------------------------------------
template <int VT>
__global__ void __launch_bounds__(MC_THREADS, 3)
mm_chunk_out_kernel(const bf16* __restrict__ q, long long ldq, const bf16* __restrict__ k,
                    long long ldk, const bf16* __restrict__ v, long long ldv,
                    const float* __restrict__ gates, const int* __restrict__ cu_q,
                    const float* __restrict__ scr_s, const float* __restrict__ scr_n,
                    float* __restrict__ num, float* __restrict__ nq, int T, int H, int K, int V,
                    int s0, float q_scale, int vec_q, int vec_k, int vec_v, MmFinish fin) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ float G[MC_L], put[MC_L];
  const int Kp = (K + 15) & ~15, Vp = (V + 7) & ~7;
  const int pk = Kp + 8, pv = VT + 8;
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);        // [MC_L][pk]
  bf16* k_s = q_s + MC_L * pk;                          // [MC_L][pk]
  bf16* v_s = k_s + MC_L * pk;                          // [MC_L][pv]
  bf16* s_hi = v_s + MC_L * pv;                         // [Kp][pv]
  bf16* s_lo = s_hi + Kp * pv;                          // [Kp][pv]
  float* n_s = reinterpret_cast<float*>(s_lo + Kp * pv);  // [Kp]
  const int h = blockIdx.z % H, s = s0 + blockIdx.z / H, v0 = blockIdx.x * VT;
  const McWhere at = mc_where(cu_q, s, s0, blockIdx.y);
  if (at.n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t plane = (size_t)T * H, cell = (size_t)at.entry * H + h;
  mc_load(q_s, pk, q + (size_t)at.t0 * ldq + (size_t)h * K, ldq, at.n, K, Kp, vec_q);
  mc_load(k_s, pk, k + (size_t)at.t0 * ldk + (size_t)h * K, ldk, at.n, K, Kp, vec_k);
  mc_load(v_s, pv, v + (size_t)at.t0 * ldv + (size_t)h * V + v0, ldv, at.n, min(VT, V - v0), VT,
          vec_v);
  const uint4* start = reinterpret_cast<const uint4*>(scr_s + cell * K * Vp);
  for (int i = tid; i < Kp * (VT / 4); i += MC_THREADS) {
    const int r = i / (VT / 4), c = (i % (VT / 4)) * 4;
    const bool ok = r < K && v0 + c < Vp;
    const uint4* w = ok ? start + (size_t)r * (Vp >> 2) + ((v0 + c) >> 2) : start;
    mc_async8(s_hi + r * pv + c, w, ok ? 8 : 0);
    mc_async8(s_lo + r * pv + c, reinterpret_cast<const uint2*>(w) + 1, ok ? 8 : 0);
  }
  for (int i = tid; i < Kp; i += MC_THREADS) n_s[i] = i < K ? scr_n[cell * K + i] : 0.f;
  if (warp == 0) mc_gates(G, put, gates, plane, (size_t)h * T + at.t0, at.n);
  mc_async_wait();
  __syncthreads();
  if (warp * 16 >= at.n) return;                        // (no barrier follows)
  const int g = lane >> 2, t2 = (lane & 3) * 2;
  const int ra = warp * 16 + g, rb = ra + 8;            // this thread's two tokens
  const float Ga = G[ra], Gb = G[rb];
  // scores of the warp's tokens against the chunk's tokens up to them
  float p[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) p[j][e] = 0.f;
  float o[VT / 8][4];
#pragma unroll
  for (int j = 0; j < VT / 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  const int arow = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, acol = (lane >> 4) * 8;
  for (int kk = 0; kk < Kp >> 4; ++kk) {
    unsigned a[4];
    mc_ldm4(a, mc_smem(q_s + arow * pk + kk * 16 + acol));
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      if (j <= 2 * warp + 1) {
        unsigned b[4];
        mc_ldm4(b, mc_smem(k_s + (j * 8 + (lane & 7) + ((lane >> 4) & 1) * 8) * pk + kk * 16 +
                           ((lane >> 3) & 1) * 8));
        mc_mma(p[j], a, b[0], b[1]);
        mc_mma(p[j + 1], a, b[2], b[3]);
      }
    }
    // the start state's part, both terms
    const int brow = kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int j = 0; j < VT / 8; j += 2) {
      unsigned b[4], bl[4];
      const int col = j * 8 + ((lane >> 4) & 1) * 8;
      mc_ldm4t(b, mc_smem(s_hi + brow * pv + col));
      mc_ldm4t(bl, mc_smem(s_lo + brow * pv + col));
      mc_mma(o[j], a, b[0], b[1]);
      mc_mma(o[j + 1], a, b[2], b[3]);
      mc_mma(o[j], a, bl[0], bl[1]);
      mc_mma(o[j + 1], a, bl[2], bl[3]);
    }
  }
  const float ea = expf(Ga), eb = expf(Gb);
#pragma unroll
  for (int j = 0; j < VT / 8; ++j) {
    o[j][0] *= ea; o[j][1] *= ea;
    o[j][2] *= eb; o[j][3] *= eb;
  }
  float sum_a = 0.f, sum_b = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = j * 8 + t2 + e;
      const float Gc = G[c], pc = put[c];
      p[j][e] = c <= ra ? p[j][e] * (expf(Ga - Gc) * pc) : 0.f;
      p[j][2 + e] = c <= rb ? p[j][2 + e] * (expf(Gb - Gc) * pc) : 0.f;
      sum_a += p[j][e];
      sum_b += p[j][2 + e];
    }
  }
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    if (kk > warp) break;
    unsigned a[4], al[4];
    a[0] = mc_pack(p[2 * kk][0], p[2 * kk][1]);
    a[1] = mc_pack(p[2 * kk][2], p[2 * kk][3]);
    a[2] = mc_pack(p[2 * kk + 1][0], p[2 * kk + 1][1]);
    a[3] = mc_pack(p[2 * kk + 1][2], p[2 * kk + 1][3]);
    al[0] = mc_pack_rest(p[2 * kk][0], p[2 * kk][1], a[0]);
    al[1] = mc_pack_rest(p[2 * kk][2], p[2 * kk][3], a[1]);
    al[2] = mc_pack_rest(p[2 * kk + 1][0], p[2 * kk + 1][1], a[2]);
    al[3] = mc_pack_rest(p[2 * kk + 1][2], p[2 * kk + 1][3], a[3]);
    const int brow = kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int j = 0; j < VT / 8; j += 2) {
      unsigned b[4];
      mc_ldm4t(b, mc_smem(v_s + brow * pv + j * 8 + ((lane >> 4) & 1) * 8));
      mc_mma(o[j], a, b[0], b[1]);
      mc_mma(o[j + 1], a, b[2], b[3]);
      mc_mma(o[j], al, b[0], b[1]);
      mc_mma(o[j + 1], al, b[2], b[3]);
    }
  }
  if (blockIdx.x == 0) {
    // n_start . q of the two tokens, the quad's lanes sharing the entries
    float da = 0.f, db = 0.f;
    for (int c = (lane & 3); c < K; c += 4) {
      da = fmaf(__bfloat162float(q_s[ra * pk + c]), n_s[c], da);
      db = fmaf(__bfloat162float(q_s[rb * pk + c]), n_s[c], db);
    }
    sum_a = fmaf(ea, da, sum_a);
    sum_b = fmaf(eb, db, sum_b);
    sum_a += __shfl_xor_sync(0xffffffffu, sum_a, 1);
    sum_a += __shfl_xor_sync(0xffffffffu, sum_a, 2);
    sum_b += __shfl_xor_sync(0xffffffffu, sum_b, 1);
    sum_b += __shfl_xor_sync(0xffffffffu, sum_b, 2);
    if (!fin.gain && (lane & 3) == 0) {
      if (ra < at.n) nq[(size_t)(at.t0 + ra) * H + h] = sum_a * q_scale;
      if (rb < at.n) nq[(size_t)(at.t0 + rb) * H + h] = sum_b * q_scale;
    }
  }
  if (fin.gain) {        // one tile holds the head's whole output
    const size_t fa = (size_t)(at.t0 + min(ra, at.n - 1)), fb = (size_t)(at.t0 + min(rb, at.n - 1));
    const float da = q_scale / (fmaxf(fabsf(sum_a * q_scale), gates[2 * plane + (size_t)h * T + fa]) +
                                fin.den_eps);
    const float db = q_scale / (fmaxf(fabsf(sum_b * q_scale), gates[2 * plane + (size_t)h * T + fb]) +
                                fin.den_eps);
    float qa = 0.f, qb = 0.f;
#pragma unroll
    for (int j = 0; j < VT / 8; ++j) {       // columns beyond V are zero
      o[j][0] *= da; o[j][1] *= da;
      o[j][2] *= db; o[j][3] *= db;
      qa += o[j][0] * o[j][0] + o[j][1] * o[j][1];
      qb += o[j][2] * o[j][2] + o[j][3] * o[j][3];
    }
    qa += __shfl_xor_sync(0xffffffffu, qa, 1);
    qa += __shfl_xor_sync(0xffffffffu, qa, 2);
    qb += __shfl_xor_sync(0xffffffffu, qb, 1);
    qb += __shfl_xor_sync(0xffffffffu, qb, 2);
    const float ia = 1.0f / sqrtf(qa / (float)V + fin.eps), ib = 1.0f / sqrtf(qb / (float)V + fin.eps);
    const bf16* gate = reinterpret_cast<const bf16*>(fin.gate) + (size_t)h * V;
    bf16* dst = reinterpret_cast<bf16*>(fin.out) + (size_t)h * V;
    const float* gain = fin.gain + (size_t)h * V;
    const size_t width = (size_t)H * V;
    const bool two = (V & 1) == 0 && (fin.gate_ld & 1) == 0 &&
                     (((uintptr_t)fin.gate | (uintptr_t)fin.out) & 3) == 0;
#pragma unroll
    for (int j = 0; j < VT / 8; ++j) {
      const int c = j * 8 + t2;
      if (c >= V) continue;
      if (two) {
        const __nv_bfloat162 za = *reinterpret_cast<const __nv_bfloat162*>(gate + fa * fin.gate_ld + c);
        const __nv_bfloat162 zb = *reinterpret_cast<const __nv_bfloat162*>(gate + fb * fin.gate_ld + c);
        const float g0 = gain[c], g1 = gain[c + 1];
        if (ra < at.n)
          *reinterpret_cast<unsigned*>(dst + fa * width + c) =
              mc_pack(o[j][0] * ia * g0 / (1.0f + expf(-__low2float(za))),
                      o[j][1] * ia * g1 / (1.0f + expf(-__high2float(za))));
        if (rb < at.n)
          *reinterpret_cast<unsigned*>(dst + fb * width + c) =
              mc_pack(o[j][2] * ib * g0 / (1.0f + expf(-__low2float(zb))),
                      o[j][3] * ib * g1 / (1.0f + expf(-__high2float(zb))));
      } else {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (c + e >= V) continue;
          const float za = __bfloat162float(gate[fa * fin.gate_ld + c + e]);
          const float zb = __bfloat162float(gate[fb * fin.gate_ld + c + e]);
          if (ra < at.n)
            dst[fa * width + c + e] =
                __float2bfloat16_rn(o[j][e] * ia * gain[c + e] / (1.0f + expf(-za)));
          if (rb < at.n)
            dst[fb * width + c + e] =
                __float2bfloat16_rn(o[j][2 + e] * ib * gain[c + e] / (1.0f + expf(-zb)));
        }
      }
    }
    return;
  }
  float* oa = num + ((size_t)(at.t0 + ra) * H + h) * V;
  float* ob = num + ((size_t)(at.t0 + rb) * H + h) * V;
  const bool pairs = (V & 1) == 0;
#pragma unroll
  for (int j = 0; j < VT / 8; ++j) {
    const int c = v0 + j * 8 + t2;
    if (pairs) {
      if (c < V && ra < at.n)
        *reinterpret_cast<float2*>(oa + c) = make_float2(o[j][0] * q_scale, o[j][1] * q_scale);
      if (c < V && rb < at.n)
        *reinterpret_cast<float2*>(ob + c) = make_float2(o[j][2] * q_scale, o[j][3] * q_scale);
    } else {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (c + e < V && ra < at.n) oa[c + e] = o[j][e] * q_scale;
        if (c + e < V && rb < at.n) ob[c + e] = o[j][2 + e] * q_scale;
      }
    }
  }
}

#define MC_MAX_K 256
IX_API int ix_mm_chunks_applies(int K, int V) { return K > 0 && K <= MC_MAX_K && V > 0; }

static inline long long mc_cells(int T, int S, int H) {
  return (long long)(T / MC_L + S + 1) * H;
}

// Floats of scratch for S sequences that bring T tokens together.
IX_API long long ix_mm_chunks_scratch_floats(int T, int S, int H, int K, int V) {
  const long long cells = mc_cells(T, S, H);
  return cells * K * ((V + 7) & ~7) + cells * K + cells + 8;
}

// Sequences s0 .. S - 1, `tokens` of them all together, the longest of max_q tokens.  num and nq,
// or, with `gain` (V at most 128), the finished rows in `out` (MmFinish).
IX_API int ix_mm_chunks(const void* q, long long ldq, const void* k, long long ldk,
                        const void* v, long long ldv, const float* gates, float* S_state,
                        float* N, const int* cu_q, const int* state_slot, float* num, float* nq,
                        int T, int tokens, int S, int s0, int max_q, int H, int K, int V,
                        float q_scale, float* scratch, const float* gain, const void* gate,
                        long long gate_ld, float eps, float den_eps, void* out,
                        cudaStream_t stream) {
  if (gain && (V > 128 || !gate || !out)) return IX_ERR_UNSUPPORTED;
  const MmFinish fin = {gain, gate, gate_ld, eps, den_eps, out};
  const int seqs = S - s0;
  if (seqs <= 0 || tokens <= 0) return IX_OK;
  if (s0 < 0 || H <= 0 || K <= 0 || K > MC_MAX_K || V <= 0 || max_q <= 0 || !scratch)
    return IX_ERR_SIZE;
  if ((uintptr_t)scratch & 15) return IX_ERR_ALIGN;
  const int chunks = (max_q + MC_L - 1) / MC_L;
  if (chunks > 65535 || (long long)H * seqs > 65535) return IX_ERR_SIZE;
  const int Kp = (K + 15) & ~15, Vp = (V + 7) & ~7;
  const long long cells = mc_cells(tokens, seqs, H);
  float* scr_s = scratch;
  float* scr_n = scr_s + cells * K * Vp;
  float* scr_p = scr_n + cells * K;
  const auto on16 = [](const void* p, long long ld, int n) {
    return ((uintptr_t)p & 15) == 0 && ld % 8 == 0 && n % 8 == 0 ? 1 : 0;
  };
  const int vq = on16(q, ldq, K), vk = on16(k, ldk, K), vv = on16(v, ldv, V);
#define MC_GO(VT)                                                                              \
  do {                                                                                         \
    const dim3 grid((V + VT - 1) / VT, chunks, H * seqs);                                      \
    const size_t own = (size_t)MC_L * (2 * (Kp + 8) + VT + 8) * 2;                             \
    const size_t tail = ((size_t)MC_L * (2 * (Kp + 8) + VT + 8) + (size_t)2 * Kp * (VT + 8)) * 2 \
                       + (size_t)Kp * 4;                                                       \
    cudaError_t e = cudaFuncSetAttribute(mm_chunk_own_kernel<VT>,                              \
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)own); \
    if (e == cudaSuccess)                                                                      \
      e = cudaFuncSetAttribute(mm_chunk_out_kernel<VT>,                                        \
                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)tail);        \
    if (e != cudaSuccess) return (int)e;                                                       \
    mm_chunk_own_kernel<VT><<<grid, MC_THREADS, own, stream>>>(                                \
        (const bf16*)k, ldk, (const bf16*)v, ldv, gates, cu_q, scr_s, scr_n, scr_p, T, H, K, V, \
        s0, vk, vv);                                                                           \
    const int items = K * (Vp / 4) + K;                                                        \
    mm_chunk_join_kernel<<<dim3((items + MJ_THREADS - 1) / MJ_THREADS, H, seqs), MJ_THREADS, 0, \
                           stream>>>(scr_s, scr_n, scr_p, S_state, N, cu_q, state_slot, H, K, V, \
                                     s0);                                                      \
    mm_chunk_out_kernel<VT><<<grid, MC_THREADS, tail, stream>>>(                               \
        (const bf16*)q, ldq, (const bf16*)k, ldk, (const bf16*)v, ldv, gates, cu_q, scr_s,     \
        scr_n, num, nq, T, H, K, V, s0, q_scale, vq, vk, vv, fin);                             \
  } while (0)
  if (V <= 64) MC_GO(64);
  else MC_GO(128);
#undef MC_GO
  return ix_launch_status();
}
