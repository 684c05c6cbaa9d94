// Parts of decoders that pair attention with a gated recurrence and squash their logits.
//
//   ix_append_kv_rows   key and value rows of a projection (views of columns) into the pages
//   ix_min_gru          z = sigmoid(a + b_z), u = x + b_x, candidate c = u + shift (u >= 0) or
//                       sigmoid(u) (u < 0); S_t = (1 - z) S_(t-1) + z c entry by entry;
//                       out = S * silu(g) * out_scale.  One thread a channel (pair) for
//                       single tokens; portions of prompts are walked in pieces side by side
//                       whose affine maps S -> A S + B are joined inside the block
//   ix_softcap_rows     x <- cap * tanh(x / cap), in place, fp32
#include "attention_distance.cuh"
#include "elementwise_vec.cuh"

// ---------------------------------------------------------------------------
// key / value rows into pages.  k [T, kvh * hd] with row pitch k_ld, v likewise; caches
// [pages, kvh, page, hd or vd]; slots [T]: page * page_size + offset.
// ---------------------------------------------------------------------------
template <typename TA, int V>
__global__ void append_kv_rows_kernel(const TA* __restrict__ k, long long k_ld,
                                      const TA* __restrict__ v, long long v_ld,
                                      const int* __restrict__ slots, TA* __restrict__ kc,
                                      TA* __restrict__ vc, int T, int kvh, int hd, int vd,
                                      int page_size) {
  IX_PDL_WAIT();
  const int kw = kvh * hd / V, vw = kvh * vd / V, per = kw + vw;
  const int hk = hd / V, hv = vd / V;
  const long long total = (long long)T * per;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total;
       i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / per);
    const int c = (int)(i - (long long)t * per);
    const int slot = slots[t];
    if (slot < 0) continue;
    const int page = slot / page_size, off = slot - page * page_size;
    const bool is_v = c >= kw;
    const int cc = is_v ? c - kw : c;
    const int hw = is_v ? hv : hk;
    const int h = cc / hw, d = cc - h * hw;
    const size_t row = ((size_t)page * kvh + h) * page_size + off;
    const TA* src = is_v ? v + (size_t)t * v_ld + (size_t)cc * V : k + (size_t)t * k_ld + (size_t)cc * V;
    TA* dst = (is_v ? vc + row * vd : kc + row * hd) + (size_t)d * V;
    if (V * sizeof(TA) == 16) *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
    else
#pragma unroll
      for (int j = 0; j < V; ++j) dst[j] = src[j];
  }
}

IX_API int ix_append_kv_rows(const void* k, long long k_ld, const void* v, long long v_ld,
                             const int* slots, void* k_cache, void* v_cache, int act_dtype, int T,
                             int kvh, int hd, int vd, int page_size, cudaStream_t stream) {
  if (T <= 0) return IX_OK;
  if (kvh <= 0 || hd <= 0 || vd <= 0 || page_size <= 0 || !slots || !k_cache || !v_cache)
    return IX_ERR_SIZE;
  const int esize = act_dtype == IX_F32 ? 4 : 2, vec = 16 / esize;
  const bool wide = hd % vec == 0 && vd % vec == 0 && k_ld % vec == 0 && v_ld % vec == 0 &&
                    (((uintptr_t)k | (uintptr_t)v | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0;
  const long long items = (long long)T * kvh * (hd + vd) / (wide ? vec : 1);
  const int threads = 256;
  long long blocks = (items + threads - 1) / threads;
  if (blocks > 148 * 16) blocks = 148 * 16;
  IX_DISPATCH_DTYPE(act_dtype, TA, {
    constexpr int V = 16 / (int)sizeof(TA);
    if (wide)
      ix_launch(append_kv_rows_kernel<TA, V>, dim3((unsigned)blocks), dim3(threads), 0, stream,
                (const TA*)k, k_ld, (const TA*)v, v_ld, slots, (TA*)k_cache, (TA*)v_cache, T, kvh,
                hd, vd, page_size);
    else
      ix_launch(append_kv_rows_kernel<TA, 1>, dim3((unsigned)blocks), dim3(threads), 0, stream,
                (const TA*)k, k_ld, (const TA*)v, v_ld, slots, (TA*)k_cache, (TA*)v_cache, T, kvh,
                hd, vd, page_size);
  });
  return ix_launch_status();
}

// ---------------------------------------------------------------------------
// the gated recurrence
// ---------------------------------------------------------------------------
// The 32-bit mode takes the accurate exponential and division, bfloat16 runs the fast ones
// (an error of a few units in the last place of fp32).
template <typename TA> __device__ __forceinline__ float mg_sigmoid(float x);
template <> __device__ __forceinline__ float mg_sigmoid<float>(float x) {
  return 1.0f / (1.0f + expf(-x));
}
template <> __device__ __forceinline__ float mg_sigmoid<bf16>(float x) {
  return __fdividef(1.0f, 1.0f + __expf(-fmaxf(x, -80.f)));
}

// a token's map S -> a S + b
template <typename TA>
__device__ __forceinline__ void mg_map(float zr, float xr, float zb, float xb, float shift,
                                       float& a, float& b) {
  const float z = mg_sigmoid<TA>(zr + zb);
  const float u = xr + xb;
  const float c = u >= 0.f ? u + shift : mg_sigmoid<TA>(u);
  a = 1.0f - z;
  b = z * c;
}
template <typename TA> __device__ __forceinline__ float mg_gate(float S, float g, float scale) {
  return S * (g * mg_sigmoid<TA>(g)) * scale;
}

template <typename TA, int V> struct MgVec;
template <typename TA> struct MgVec<TA, 1> {
  static __device__ __forceinline__ void load(const TA* p, float* f) { f[0] = to_f32(p[0]); }
  static __device__ __forceinline__ void store(TA* p, const float* f) { p[0] = from_f32<TA>(f[0]); }
};
template <> struct MgVec<bf16, 2> {
  static __device__ __forceinline__ void load(const bf16* p, float* f) {
    const float2 t = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    f[0] = t.x;
    f[1] = t.y;
  }
  static __device__ __forceinline__ void store(bf16* p, const float* f) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(f[0], f[1]);
  }
};
template <> struct MgVec<float, 2> {
  static __device__ __forceinline__ void load(const float* p, float* f) {
    const float2 t = *reinterpret_cast<const float2*>(p);
    f[0] = t.x;
    f[1] = t.y;
  }
  static __device__ __forceinline__ void store(float* p, const float* f) {
    *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]);
  }
};

// single tokens: sequence s brings token cu_q[s]
template <typename TA, int V>
__global__ void min_gru_step_kernel(const TA* __restrict__ front, long long ld,
                                    const float* __restrict__ z_bias,
                                    const float* __restrict__ x_bias, float shift,
                                    float* __restrict__ state, const int* __restrict__ slots,
                                    const int* __restrict__ cu_q, TA* __restrict__ out,
                                    long long o_ld, float out_scale, int W) {
  IX_PDL_WAIT();
  const int s = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= W) return;
  const int t = cu_q[s];
  const TA* row = front + (size_t)t * ld;
  float* st = state + (size_t)slots[s] * W + c;
  float z[V], x[V], g[V], y[V];
  MgVec<TA, V>::load(row + c, z);
  MgVec<TA, V>::load(row + W + c, x);
  MgVec<TA, V>::load(row + 2 * W + c, g);
#pragma unroll
  for (int i = 0; i < V; ++i) {
    float a, b;
    mg_map<TA>(z[i], x[i], z_bias[c + i], x_bias[c + i], shift, a, b);
    const float S = fmaf(a, st[i], b);
    st[i] = S;
    y[i] = mg_gate<TA>(S, g[i], out_scale);
  }
  MgVec<TA, V>::store(out + (size_t)t * o_ld + c, y);
}

// Portions: a block owns CL * V neighbouring channels of one sequence; its threads are CL
// channel lanes times NW * 32 / CL time lanes, a time lane MG_L neighbouring tokens of a
// stretch.  Every thread forms the map of its tokens, the maps of the time lanes before it
// are joined (shuffles inside a warp, shared memory between warps), and the thread walks its
// tokens from the state it then knows.
//   MODE 0: the block takes the whole portion, stretch by stretch (portions of a few
//           hundred tokens: narrow tiles of channels, many time lanes);
//   MODE 1: long portions are cut into segments of seg_len tokens, blockIdx.z picks one; the
//           map of the segment alone goes to maps[s][1 + segment] as (A, B) per channel, and
//           the state ahead of the portion to maps[s][0] as (0, S);
//   MODE 2: the segment's block joins the maps ahead of it and walks its tokens.
// z and x are read twice then, the second time from L2, and the segments fill the device.
#define MG_L 8

template <typename TA, int V, int CL, int NW, int MODE>
__global__ void __launch_bounds__(NW * 32)
min_gru_scan_kernel(const TA* __restrict__ front, long long ld, const float* __restrict__ z_bias,
                    const float* __restrict__ x_bias, float shift, float* __restrict__ state,
                    const int* __restrict__ slots, const int* __restrict__ cu_q,
                    TA* __restrict__ out, long long o_ld, float out_scale, int W, int seg_len,
                    int segments, float2* __restrict__ maps) {
  constexpr int CH = CL * V;                    // channels of the block
  constexpr int TW = 32 / CL;                   // time lanes of a warp
  constexpr int SPAN = NW * TW * MG_L;          // tokens of a stretch
  __shared__ float wa[NW][CH], wb[NW][CH];
  __shared__ float carry[CH], carry_a[CH];
  IX_PDL_WAIT();
  const int s = blockIdx.y;
  const int tok0 = cu_q[s], total = cu_q[s + 1] - tok0;
  const int first = MODE == 0 ? 0 : (int)blockIdx.z * seg_len;
  const int n = MODE == 0 ? total : min(total, first + seg_len);
  if (first >= n) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int cl = lane % CL, tw = lane / CL;
  const int tl = warp * TW + tw;
  const int c0 = blockIdx.x * CH;
  const int c = c0 + cl * V;
  const bool live = c < W;                      // W is a multiple of V
  float* st = state + (size_t)slots[s] * W;
  float2* my_maps = MODE == 0 ? nullptr : maps + (size_t)s * (segments + 1) * W;
  for (int i = threadIdx.x; i < CH; i += NW * 32) {
    const bool ok = c0 + i < W;
    float x = 0.f;
    if (MODE == 0 && ok) x = st[c0 + i];
    if (MODE == 1 && blockIdx.z == 0 && ok) my_maps[c0 + i] = make_float2(0.f, st[c0 + i]);
    if (MODE == 2 && ok) {
#pragma unroll 4
      for (int g = 0; g <= (int)blockIdx.z; ++g) {
        const float2 m = my_maps[(size_t)g * W + c0 + i];
        x = fmaf(m.x, x, m.y);
      }
    }
    carry[i] = x;                               // MODE 1: B of what came before, A beside it
    if (MODE == 1) carry_a[i] = 1.f;
  }
  float zb[V], xb[V];
#pragma unroll
  for (int i = 0; i < V; ++i) {
    zb[i] = live ? z_bias[c + i] : 0.f;
    xb[i] = live ? x_bias[c + i] : 0.f;
  }
  for (int base = first; base < n; base += SPAN) {
    const int t0 = base + tl * MG_L;
    const int m = live ? max(0, min(MG_L, n - t0)) : 0;
    // Loads and maps without a branch, so that all loads are out before the first is used:
    // tokens past the end and channels past the width read a valid place and count as the
    // identity map.
    const TA* row = front + (size_t)tok0 * ld + (live ? c : 0);
    float a[MG_L][V], b[MG_L][V], g[MODE == 1 ? 1 : MG_L][V];
#pragma unroll
    for (int i = 0; i < MG_L; ++i) {
      const TA* p = row + (size_t)min(t0 + i, n - 1) * ld;
      MgVec<TA, V>::load(p, a[i]);
      MgVec<TA, V>::load(p + W, b[i]);
      if (MODE != 1) MgVec<TA, V>::load(p + 2 * W, g[MODE == 1 ? 0 : i]);
    }
    float A[V], B[V];
#pragma unroll
    for (int v = 0; v < V; ++v) {
      A[v] = 1.f;
      B[v] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < MG_L; ++i)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float ma, mb;
        mg_map<TA>(a[i][v], b[i][v], zb[v], xb[v], shift, ma, mb);
        a[i][v] = i < m ? ma : 1.f;
        b[i][v] = i < m ? mb : 0.f;
        A[v] *= a[i][v];
        B[v] = fmaf(a[i][v], B[v], b[i][v]);
      }
    // inclusive maps over the warp's time lanes
#pragma unroll
    for (int o = CL; o < 32; o <<= 1)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const float pa = __shfl_up_sync(0xffffffffu, A[v], o);
        const float pb = __shfl_up_sync(0xffffffffu, B[v], o);
        if (lane >= o) {
          B[v] = fmaf(A[v], pb, B[v]);
          A[v] *= pa;
        }
      }
    if (tw == TW - 1)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        wa[warp][cl * V + v] = A[v];
        wb[warp][cl * V + v] = B[v];
      }
    if (MODE == 1) {          // the stretch's map behind the one of the stretches before
      __syncthreads();
      for (int i = threadIdx.x; i < CH; i += NW * 32) {
        float x = carry[i], y = carry_a[i];
#pragma unroll
        for (int w = 0; w < NW; ++w) {
          x = fmaf(wa[w][i], x, wb[w][i]);
          y *= wa[w][i];
        }
        carry[i] = x;
        carry_a[i] = y;
      }
      __syncthreads();
      continue;
    }
    // exclusive inside the warp
    if (TW > 1) {
#pragma unroll
      for (int v = 0; v < V; ++v) {
        A[v] = __shfl_up_sync(0xffffffffu, A[v], CL);
        B[v] = __shfl_up_sync(0xffffffffu, B[v], CL);
      }
    }
    if (tw == 0)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        A[v] = 1.f;
        B[v] = 0.f;
      }
    float S[V];
    __syncthreads();          // the warps' maps and the carried state are there
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float x = carry[cl * V + v];
      for (int w = 0; w < warp; ++w) x = fmaf(wa[w][cl * V + v], x, wb[w][cl * V + v]);
      S[v] = fmaf(A[v], x, B[v]);
    }
    TA* o = out + (size_t)(tok0 + t0) * o_ld + c;
#pragma unroll
    for (int i = 0; i < MG_L; ++i) {
      float y[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        S[v] = fmaf(a[i][v], S[v], b[i][v]);
        y[v] = mg_gate<TA>(S[v], g[MODE == 1 ? 0 : i][v], out_scale);
      }
      if (i < m) MgVec<TA, V>::store(o + (size_t)i * o_ld, y);
    }
    __syncthreads();          // everyone has read the carried state
    // the thread of the stretch's last token knows the state behind it
    if (m > 0 && (t0 + m == n || (tl == NW * TW - 1)))
#pragma unroll
      for (int v = 0; v < V; ++v) carry[cl * V + v] = S[v];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < CH; i += NW * 32) {
    if (c0 + i >= W) break;
    if (MODE == 1) my_maps[(size_t)(blockIdx.z + 1) * W + c0 + i] = make_float2(carry_a[i], carry[i]);
    else if (n == total) st[c0 + i] = carry[i];
  }
}

#define MG_SHORT 512       // portions up to this many tokens take MODE 0
#define MG_STRETCH 64      // tokens of a stretch in MODE 1 and 2
#define MG_MAX_SEGMENTS 32

// Segments a step whose longest portion has max_q tokens is cut into (1: not cut); the scratch
// is float2 [sequences that are no single tokens][segments + 1][W].
IX_API int ix_min_gru_segments(int max_q) {
  if (max_q <= MG_SHORT) return 1;
  int len = (max_q + MG_MAX_SEGMENTS - 1) / MG_MAX_SEGMENTS;
  len = (len + MG_STRETCH - 1) / MG_STRETCH * MG_STRETCH;
  return (max_q + len - 1) / len;
}

template <typename TA, int V>
static void launch_min_gru_scan(const void* front, long long ld, const float* z_bias,
                                const float* x_bias, float shift, float* state, const int* slots,
                                const int* cu_q, void* out, long long o_ld, float out_scale,
                                int W, int S, int max_q, int segments, float* maps,
                                cudaStream_t stream) {
  if (segments <= 1) {
    constexpr int CL = 16 / V;
    ix_launch(min_gru_scan_kernel<TA, V, CL, 16, 0>, dim3((W + 15) / 16, S), dim3(512), 0, stream,
              (const TA*)front, ld, z_bias, x_bias, shift, state, slots, cu_q, (TA*)out, o_ld,
              out_scale, W, 0, 1, (float2*)nullptr);
    return;
  }
  int len = (max_q + segments - 1) / segments;
  len = (len + MG_STRETCH - 1) / MG_STRETCH * MG_STRETCH;
  const dim3 grid((W + 32 * V - 1) / (32 * V), S, segments);
  ix_launch(min_gru_scan_kernel<TA, V, 32, 8, 1>, grid, dim3(256), 0, stream, (const TA*)front, ld,
            z_bias, x_bias, shift, state, slots, cu_q, (TA*)out, o_ld, out_scale, W, len, segments,
            (float2*)maps);
  ix_launch(min_gru_scan_kernel<TA, V, 32, 8, 2>, grid, dim3(256), 0, stream, (const TA*)front, ld,
            z_bias, x_bias, shift, state, slots, cu_q, (TA*)out, o_ld, out_scale, W, len, segments,
            (float2*)maps);
}

// front: rows of pitch ld, columns [z: W | x: W | g: W]; state [slots, W] fp32; slots and cu_q
// are those of the S sequences; the first `singles` of them bring one token each, the longest
// of the rest max_q.  segments > 1 (see ix_min_gru_segments): maps is the scratch.
IX_API int ix_min_gru(const void* front, long long ld, const float* z_bias, const float* x_bias,
                      float shift, float* state, const int* slots, const int* cu_q, void* out,
                      long long o_ld, float out_scale, int act_dtype, int S, int singles, int W,
                      int max_q, int segments, float* maps, cudaStream_t stream) {
  if (S <= 0) return IX_OK;
  if (W <= 0 || singles < 0 || singles > S || S > 65535 || ld < 3LL * W || o_ld < W)
    return IX_ERR_SIZE;
  if (segments < 1 || (segments > 1 && (!maps || max_q <= 0 ||
                                        segments != ix_min_gru_segments(max_q))))
    return IX_ERR_SIZE;
  const int esize = act_dtype == IX_F32 ? 4 : 2;
  const bool pairs = W % 2 == 0 && ld % 2 == 0 && o_ld % 2 == 0 &&
                     (((uintptr_t)front | (uintptr_t)out) % (2 * esize)) == 0;
  const int rest = S - singles;
#define IX_MG(V)                                                                                \
  IX_DISPATCH_DTYPE(act_dtype, TA, {                                                            \
    if (singles > 0)                                                                            \
      ix_launch(min_gru_step_kernel<TA, V>, dim3((W / V + 127) / 128, singles), dim3(128), 0,   \
                stream, (const TA*)front, ld, z_bias, x_bias, shift, state, slots, cu_q,        \
                (TA*)out, o_ld, out_scale, W);                                                  \
    if (rest > 0)                                                                               \
      launch_min_gru_scan<TA, V>(front, ld, z_bias, x_bias, shift, state, slots + singles,      \
                                 cu_q + singles, out, o_ld, out_scale, W, rest, max_q, segments, \
                                 maps, stream);                                                 \
  })
  if (pairs) IX_MG(2);
  else IX_MG(1);
#undef IX_MG
  return ix_launch_status();
}

// ---------------------------------------------------------------------------
// squashed logits
// ---------------------------------------------------------------------------
__global__ void softcap_rows_kernel(float* __restrict__ x, long long n4, long long n, float cap) {
  IX_PDL_WAIT();
  float4* x4 = reinterpret_cast<float4*>(x);
  const long long step = (long long)gridDim.x * blockDim.x;
  const long long first = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  for (long long i = first; i < n4; i += step) {
    float4 v = x4[i];
    v.x = cap * tanhf(v.x / cap);
    v.y = cap * tanhf(v.y / cap);
    v.z = cap * tanhf(v.z / cap);
    v.w = cap * tanhf(v.w / cap);
    x4[i] = v;
  }
  for (long long i = 4 * n4 + first; i < n; i += step) x[i] = cap * tanhf(x[i] / cap);
}

IX_API int ix_softcap_rows(float* x, long long n, float cap, cudaStream_t stream) {
  if (n <= 0) return IX_OK;
  if (!(cap > 0.f)) return IX_ERR_SIZE;
  const long long n4 = ((uintptr_t)x & 15) == 0 ? n / 4 : 0;
  long long blocks = ((n4 > 0 ? n4 : n) + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  ix_launch(softcap_rows_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, n4, n, cap);
  return ix_launch_status();
}
