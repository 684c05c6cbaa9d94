// Several residual streams beside each other, and the elementwise norm.
//
// A decoder may carry n streams x_1 .. x_n per token instead of one.  A sublayer reads
// u = sum_s read[s] x_s, and its output y enters by x_t <- sum_s mix[s, t] x_s + put[t] y,
// all streams at once from the old ones.  The update of one sublayer and the reading of the
// next are one pass over the streams here (ix_stream_step), together with
//  * what y still is: a plain row, or a mixture's expert rows with their weights and the
//    shared expert's part, combined on the fly;
//  * the norm of u: tanh(alpha u) gain + bias entry by entry (no mean, no variance), or
//    none (u itself in fp32, for a norm that needs the whole row).
// A plain residual stream is the case n = 1, mix = put = read = 1.
//
// Streams are fp32 [T, n, W]; all arithmetic is fp32 with the accurate tanhf.  A thread owns
// VW neighbouring entries of a column and walks the tokens, so the constants are read once.
#include "common.cuh"
#include "elementwise_vec.cuh"

#define ST_THREADS 128
#define ST_MAX_STREAMS 16

struct StCombine {          // a mixture's output that was not written: see moe_combine
  const void* rows;         // grouped expert rows [A, W] (null: y is a plain row)
  const int* dest;          // [T, k] row of each assignment
  const float* weight;      // [T, k], or null: the plain sum
  const void* shared;       // [T, W] or null
  const float* shared_logit;  // [T] or null (ungated)
  int k;
};

template <int VW> struct StVec { float v[VW]; };

template <int VW>
__device__ __forceinline__ StVec<VW> st_load(const float* p) {
  StVec<VW> r;
  if (VW == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    r.v[0] = a.x; r.v[VW > 1 ? 1 : 0] = a.y; r.v[VW > 2 ? 2 : 0] = a.z; r.v[VW > 3 ? 3 : 0] = a.w;
  } else {
    r.v[0] = p[0];
  }
  return r;
}
template <int VW>
__device__ __forceinline__ StVec<VW> st_load(const bf16* p) {
  StVec<VW> r;
  if (VW == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.y));
    r.v[0] = lo.x; r.v[VW > 1 ? 1 : 0] = lo.y; r.v[VW > 2 ? 2 : 0] = hi.x; r.v[VW > 3 ? 3 : 0] = hi.y;
  } else {
    r.v[0] = __bfloat162float(p[0]);
  }
  return r;
}
template <int VW>
__device__ __forceinline__ void st_store(float* p, const StVec<VW>& r) {
  if (VW == 4)
    *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[VW > 1 ? 1 : 0], r.v[VW > 2 ? 2 : 0],
                                                r.v[VW > 3 ? 3 : 0]);
  else p[0] = r.v[0];
}
template <int VW>
__device__ __forceinline__ void st_store(bf16* p, const StVec<VW>& r) {
  if (VW == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[VW > 1 ? 1 : 0]);
    const __nv_bfloat162 hi = __floats2bfloat162_rn(r.v[VW > 2 ? 2 : 0], r.v[VW > 3 ? 3 : 0]);
    uint2 a;
    a.x = *reinterpret_cast<const unsigned*>(&lo);
    a.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = a;
  } else {
    p[0] = __float2bfloat16_rn(r.v[0]);
  }
}

// FIXED: n == NS; otherwise n <= NS.  With FIXED and a plain y the constants live in registers;
// they are read from shared memory otherwise: combining a mixture's rows is a chain of
// dependent reads (row numbers, then rows), for which more threads in flight are worth more.
template <int NS, bool FIXED, bool COMBINE, int VW, typename TY, typename TO>
__global__ void __launch_bounds__(ST_THREADS)
stream_step_kernel(float* __restrict__ streams, const TY* __restrict__ y, StCombine cmb,
                   const float* __restrict__ mix, const float* __restrict__ put,
                   const float* __restrict__ read, const float* __restrict__ alpha_p,
                   const float* __restrict__ gain, const float* __restrict__ bias,
                   const int* __restrict__ rows, TO* __restrict__ out, int R, int W, int n,
                   int write_back) {
  __shared__ float mix_s[NS * NS], put_s[NS], read_s[NS];
  IX_PDL_WAIT();
  const bool updates = mix != nullptr;
  for (int i = threadIdx.x; i < n * n; i += ST_THREADS)
    mix_s[i] = updates ? mix[i] : (i / n == i % n ? 1.f : 0.f);
  for (int i = threadIdx.x; i < n; i += ST_THREADS) {
    put_s[i] = updates ? put[i] : 0.f;
    read_s[i] = read[i];
  }
  __syncthreads();
  const int c = (blockIdx.x * ST_THREADS + threadIdx.x) * VW;
  if (c >= W) return;
  constexpr bool REGS = FIXED && !COMBINE;
  float mr[REGS ? NS * NS : 1], pr[REGS ? NS : 1], rr[REGS ? NS : 1];
  if (REGS) {
#pragma unroll
    for (int i = 0; i < (REGS ? NS * NS : 1); ++i) mr[i] = mix_s[i];
#pragma unroll
    for (int i = 0; i < (REGS ? NS : 1); ++i) {
      pr[i] = put_s[i];
      rr[i] = read_s[i];
    }
  }
  StVec<VW> g, b;
  float alpha = 0.f;
  if (gain) {
    alpha = alpha_p[0];
    g = st_load<VW>(gain + c);
    b = st_load<VW>(bias + c);
  }
  for (int r = blockIdx.y; r < R; r += gridDim.y) {
    const size_t t = rows ? (size_t)rows[r] : (size_t)r;
    float* x = streams + t * n * W + c;
    StVec<VW> old[NS], d;
#pragma unroll
    for (int e = 0; e < VW; ++e) d.v[e] = 0.f;
    if (COMBINE) {
      // four assignments at a time, without a branch between their reads: row numbers and
      // weights, then the rows
      const TY* er = reinterpret_cast<const TY*>(cmb.rows);
      const int* dest = cmb.dest + t * cmb.k;
      const float* weight = cmb.weight ? cmb.weight + t * cmb.k : read;
      const float sg = cmb.shared && cmb.shared_logit
                           ? 1.0f / (1.0f + expf(-cmb.shared_logit[t])) : 1.0f;
      for (int j0 = 0; j0 < cmb.k; j0 += 4) {
        int row[4];
        float w[4];
        StVec<VW> f[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int a = min(j0 + j, cmb.k - 1);
          row[j] = dest[a];
          w[j] = weight[cmb.weight ? a : 0];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) f[j] = st_load<VW>(er + (size_t)row[j] * W + c);
        if (j0 == 0) {
#pragma unroll
          for (int s = 0; s < NS; ++s)
            if (FIXED || s < n) old[s] = st_load<VW>(x + (size_t)s * W);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float wj = j0 + j < cmb.k ? (cmb.weight ? w[j] : 1.0f) : 0.f;
#pragma unroll
          for (int e = 0; e < VW; ++e) d.v[e] = fmaf(wj, f[j].v[e], d.v[e]);
        }
      }
      if (cmb.shared) {
        const StVec<VW> f = st_load<VW>(reinterpret_cast<const TY*>(cmb.shared) + t * W + c);
#pragma unroll
        for (int e = 0; e < VW; ++e) d.v[e] = fmaf(sg, f.v[e], d.v[e]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < NS; ++s)
        if (FIXED || s < n) old[s] = st_load<VW>(x + (size_t)s * W);
      if (updates) d = st_load<VW>(y + t * W + c);
    }
    StVec<VW> u;
#pragma unroll
    for (int e = 0; e < VW; ++e) u.v[e] = 0.f;
#pragma unroll(FIXED ? NS : 1)
    for (int o = 0; o < NS; ++o) {
      if (!FIXED && o >= n) break;
      StVec<VW> v;
      if (updates) {
        const float po = REGS ? pr[REGS ? o : 0] : put_s[o];
#pragma unroll
        for (int e = 0; e < VW; ++e) v.v[e] = po * d.v[e];
#pragma unroll
        for (int s = 0; s < NS; ++s) {
          if (!FIXED && s >= n) break;
          const float m = REGS ? mr[REGS ? s * NS + o : 0] : mix_s[s * n + o];
#pragma unroll
          for (int e = 0; e < VW; ++e) v.v[e] = fmaf(m, old[s].v[e], v.v[e]);
        }
        if (write_back) st_store<VW>(x + (size_t)o * W, v);
      } else {
        v = old[o];
      }
      const float ro = REGS ? rr[REGS ? o : 0] : read_s[o];
#pragma unroll
      for (int e = 0; e < VW; ++e) u.v[e] = fmaf(ro, v.v[e], u.v[e]);
    }
    if (gain) {
#pragma unroll
      for (int e = 0; e < VW; ++e) u.v[e] = fmaf(tanhf(alpha * u.v[e]), g.v[e], b.v[e]);
    }
    st_store<VW>(out + (size_t)r * W + c, u);
  }
}

IX_API int ix_stream_max() { return ST_MAX_STREAMS; }

// streams fp32 [*, n, W].  mix [n, n] (from, to) and put [n]: the update by y (null: none; the
// streams stay).  y: [*, W] of y_dtype, or null with the combine arguments (expert rows of
// y_dtype).  read [n].  gain, bias [W] and alpha (one number): the norm; gain null: `out` is
// the read row itself, fp32.  rows: R rows to gather (the streams are then not written), or
// null: all R tokens.
IX_API int ix_stream_step(float* streams, const void* y, int y_dtype, const void* c_rows,
                          const int* c_dest, const float* c_weight, const void* c_shared,
                          const float* c_logit, int c_k, const float* mix, const float* put,
                          const float* read, const float* alpha, const float* gain,
                          const float* bias, const int* rows, void* out, int out_dtype, int R,
                          int W, int n, int write_back, cudaStream_t stream) {
  if (R <= 0) return IX_OK;
  if (W <= 0 || n <= 0 || n > ST_MAX_STREAMS || !read) return IX_ERR_SIZE;
  if ((mix == nullptr) != (put == nullptr) || (mix && !y && !c_rows) ||
      (gain && (!alpha || !bias)) || (!gain && out_dtype != IX_F32))
    return IX_ERR_SIZE;
  if (c_rows && (c_k <= 0 || !c_dest)) return IX_ERR_SIZE;
  const StCombine cmb = {c_rows, c_dest, c_weight, c_shared, c_logit, c_k};
  const size_t ya = y_dtype == IX_F32 ? 16 : 8, oa = out_dtype == IX_F32 ? 16 : 8;
  const bool vec = W % 4 == 0 &&
                   (((uintptr_t)streams | (uintptr_t)gain | (uintptr_t)bias) & 15) == 0 &&
                   (((uintptr_t)y | (uintptr_t)c_rows | (uintptr_t)c_shared) % ya) == 0 &&
                   ((uintptr_t)out % oa) == 0;
  const int cols = (W / (vec ? 4 : 1) + ST_THREADS - 1) / ST_THREADS;
  const int colsx = vec ? cols : (W + ST_THREADS - 1) / ST_THREADS;
  // about two rounds of resident blocks: a thread's constants serve several tokens
  int by = (148 * 16 + colsx - 1) / colsx;
  if (by > R) by = R;
  if (by > 65535) by = 65535;
  const dim3 grid(colsx, by);
#define ST_GO(NS, FIXED, VW)                                                                    \
  do {                                                                                          \
    auto kern = mix && c_rows ? stream_step_kernel<NS, FIXED, true, VW, TY, TO>                 \
                              : stream_step_kernel<NS, FIXED, false, VW, TY, TO>;               \
    ix_launch(kern, grid, dim3(ST_THREADS), 0, stream, streams, (const TY*)y, cmb, mix, put,    \
              read, alpha, gain, bias, rows, (TO*)out, R, W, n, write_back);                    \
  } while (0)
#define ST_N(VW)                                                                                \
  do {                                                                                          \
    if (n == 1) ST_GO(1, true, VW);                                                             \
    else if (n == 2) ST_GO(2, true, VW);                                                        \
    else if (n == 3) ST_GO(3, true, VW);                                                        \
    else if (n == 4) ST_GO(4, true, VW);                                                        \
    else if (n <= 8) ST_GO(8, false, VW);                                                       \
    else ST_GO(16, false, VW);                                                                  \
  } while (0)
  IX_DISPATCH_DTYPE(y_dtype, TY, {
    IX_DISPATCH_DTYPE(out_dtype, TO, {
      if (vec) ST_N(4);
      else ST_N(1);
    });
  });
#undef ST_N
#undef ST_GO
  return ix_launch_status();
}

// streams[t, s] = table[ids[t]] for every s < n, widened to fp32.
template <typename TW>
__global__ void embed_streams_kernel(const TW* __restrict__ table, const int* __restrict__ ids,
                                     float* __restrict__ out, int W, int n) {
  IX_PDL_WAIT();
  const int t = blockIdx.x;
  const TW* src = table + (size_t)ids[t] * W;
  float* dst = out + (size_t)t * n * W;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < W; i += gridDim.y * blockDim.x) {
    const float v = to_f32(src[i]);
    for (int s = 0; s < n; ++s) dst[(size_t)s * W + i] = v;
  }
}

IX_API int ix_embed_streams(const void* table, int dtype, const int* ids, float* out, int T,
                            int W, int n, cudaStream_t stream) {
  if (T <= 0) return IX_OK;
  if (W <= 0 || n <= 0) return IX_ERR_SIZE;
  const int by = T >= 1024 ? 1 : (W + 255) / 256;
  IX_DISPATCH_DTYPE(dtype, TW,
                    ix_launch(embed_streams_kernel<TW>, dim3(T, by), dim3(256), 0, stream,
                              (const TW*)table, ids, out, W, n));
  return ix_launch_status();
}
