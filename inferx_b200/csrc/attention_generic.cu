// Paged causal attention with grouped KV heads and an optional sliding window,
// for any mix of prompt portions and single decoded tokens in one launch.
// This is the general kernel: any head size up to 512 (the values' may differ from the
// keys'), any element type, fp32
// arithmetic throughout with the accurate expf.  It is the whole attention of
// the 32-bit path and the fallback of the bfloat16 path for shapes the tuned
// kernels refuse.
//
// Reference behaviour: PagedAttentionKernel / PagedAttentionWithLseKernel
// (src/backends/cuda/ops/layers.cu:256-318, 329-407): query at position p of a
// sequence sees keys max(0, p-window+1)..p (all of 0..p without a window),
// score = (q.k) * scale, softmax with max subtraction, kv head = head / group.
// Unlike the reference there is no cap on the number of keys: scores are
// consumed in tiles of 128 keys with an online softmax.  One block owns one
// (token, head); its arithmetic depends only on that token's own keys, never on
// what else is in the batch or on which pages hold the keys.
//
// Two options of windowed attention: `keep_first` > 0 keeps the sequence's first
// keep_first keys visible beside the window (they are walked first, as if they stood
// directly before the window), and a sink per head joins the softmax's denominator (a
// key of that score that has no value); IxRows has it, and a gate per (token, head).
//
// A third form (attention_distance.cuh) multiplies a score by its head's temperature, takes
// r1 ln(1 + r2 distance) off and may confine a query to its own run of positions.
#include "attention_distance.cuh"

#define ATT_TILE 128
#define ATT_THREADS 128
#define ATT_MAX_DPT 4  // dims per thread: head_dim <= ATT_THREADS * ATT_MAX_DPT

template <typename TA>
__global__ void __launch_bounds__(ATT_THREADS)
paged_attention_generic_kernel(const TA* __restrict__ q, const TA* __restrict__ kc,
                               const TA* __restrict__ vc, const int* __restrict__ block_table,
                               const int* __restrict__ seq_of_token,
                               const int* __restrict__ positions, TA* __restrict__ out, int heads,
                               int kvh, int hd, int vd, int page_size, int max_blocks,
                               int window, float scale, float softcap, int keep_first,
                               IxRows rows, IxDistance dist) {
  extern __shared__ float smem[];
  float* qs = smem;        // [hd]
  float* sc = smem + hd;   // [ATT_TILE]
  const int t = blockIdx.x;
  const int h = blockIdx.y;
  const int s = seq_of_token[t];
  const int pos = positions[t];
  const int kh = h / (heads / kvh);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = ATT_THREADS / 32;
  const int* bt = block_table + (size_t)s * max_blocks;

  const TA* qrow = q + (size_t)t * rows.q_ld + (size_t)h * hd;
  const bool far = dist.temp != nullptr;
  const float temp = far ? dist.temp[h] : 1.f;
  const float r1 = far ? dist.r1[h] : 0.f, r2 = far ? dist.r2[h] : 0.f;
  for (int d = threadIdx.x; d < hd; d += ATT_THREADS) qs[d] = to_f32(qrow[d]);
  __syncthreads();

  float acc[ATT_MAX_DPT];
#pragma unroll
  for (int i = 0; i < ATT_MAX_DPT; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;

  const int start = ix_first_key(pos, window, dist.chunk);
  // the kept first keys count as positions start - kept .. start - 1 of the walk
  const int kept = min(keep_first, start);
  for (int tile0 = start - kept; tile0 <= pos; tile0 += ATT_TILE) {
    const int n = min(ATT_TILE, pos + 1 - tile0);
    // scores: one warp per key, lanes over the head dimension
    for (int j = warp; j < n; j += nwarps) {
      const int kw = tile0 + j;
      const int kp = kw < start ? kw - (start - kept) : kw;
      const int page = bt[kp / page_size];
      const int off = kp % page_size;
      const TA* krow = kc + (((size_t)page * kvh + kh) * page_size + off) * hd;
      float dot = 0.f;
      for (int d = lane; d < hd; d += 32) dot += qs[d] * to_f32(krow[d]);
      dot = warp_sum(dot);
      if (lane == 0) {
        float sv = dot * scale;
        if (far) sv = sv * temp - r1 * log1pf(r2 * (float)(pos - kp));
        sc[j] = softcap > 0.f ? softcap * tanhf(sv / softcap) : sv;   // squashed scores
      }
    }
    __syncthreads();
    float tm = -INFINITY;
    for (int j = 0; j < n; ++j) tm = fmaxf(tm, sc[j]);
    const float m_new = fmaxf(m, tm);
    const float corr = expf(m - m_new);  // 0 on the first tile (m = -inf)
    __syncthreads();
    for (int j = threadIdx.x; j < n; j += ATT_THREADS) sc[j] = expf(sc[j] - m_new);
    __syncthreads();
    float psum = 0.f;
    for (int j = 0; j < n; ++j) psum += sc[j];
    l = l * corr + psum;
    m = m_new;
#pragma unroll
    for (int i = 0; i < ATT_MAX_DPT; ++i) acc[i] *= corr;
    for (int j = 0; j < n; ++j) {
      const int kw = tile0 + j;
      const int kp = kw < start ? kw - (start - kept) : kw;
      const int page = bt[kp / page_size];
      const int off = kp % page_size;
      const TA* vrow = vc + (((size_t)page * kvh + kh) * page_size + off) * vd;
      const float p = sc[j];
#pragma unroll
      for (int i = 0; i < ATT_MAX_DPT; ++i) {
        const int d = threadIdx.x + i * ATT_THREADS;
        if (d < vd) acc[i] += p * to_f32(vrow[d]);
      }
    }
    __syncthreads();
  }
  TA* orow = out + (size_t)t * rows.o_ld + (size_t)h * vd;
  float inv_l = 1.0f / l;
  if (rows.sink) {     // one more term, exp(sink - max), in the denominator
    const float sk = rows.sink[h];
    const float top = fmaxf(m, sk);
    const float c = expf(m - top);
    inv_l = c / (l * c + expf(sk - top));
  }
  const float factor = ix_result_factor<TA>(rows, t, h);
#pragma unroll
  for (int i = 0; i < ATT_MAX_DPT; ++i) {
    const int d = threadIdx.x + i * ATT_THREADS;
    if (d < vd) orow[d] = from_f32<TA>(acc[i] * inv_l * factor);
  }
}

// The largest head size any attention kernel of this library takes (this one; the tuned
// kernels take fewer); a model is checked against it when it is built.
IX_API int ix_attention_max_head_dim() { return ATT_THREADS * ATT_MAX_DPT; }

static int generic_checked(const void* q, const void* k_cache, const void* v_cache,
                           const int* block_table, const int* seq_of_token, const int* positions,
                           void* out, int act_dtype, int T, int heads, int kvh, int hd, int vd,
                           int page_size, int max_blocks, int window, float scale, float softcap,
                           int keep_first, IxRows rows, IxDistance dist,
                           cudaStream_t stream) {
  if (T <= 0) return IX_OK;
  if (heads <= 0 || kvh <= 0 || heads % kvh != 0 || page_size <= 0 || max_blocks <= 0)
    return IX_ERR_SIZE;
  if (hd <= 0 || hd > ATT_THREADS * ATT_MAX_DPT) return IX_ERR_SIZE;
  if (vd <= 0 || vd > ATT_THREADS * ATT_MAX_DPT) return IX_ERR_SIZE;   // values of another size
  if (window < 0 || keep_first < 0) return IX_ERR_SIZE;
  const size_t smem = (size_t)(hd + ATT_TILE) * sizeof(float);
  if (heads > 65535) return IX_ERR_SIZE;
  dim3 grid(T, heads);
  IX_DISPATCH_DTYPE(act_dtype, TA,
                    (paged_attention_generic_kernel<TA><<<grid, ATT_THREADS, smem, stream>>>(
                        (const TA*)q, (const TA*)k_cache, (const TA*)v_cache, block_table,
                        seq_of_token, positions, (TA*)out, heads, kvh, hd, vd, page_size,
                        max_blocks, window, scale, softcap, keep_first, rows, dist)));
  return ix_launch_status();
}

IX_API int ix_paged_attention_generic(const void* q, const void* k_cache, const void* v_cache,
                                      const int* block_table, const int* seq_of_token,
                                      const int* positions, void* out, int act_dtype, int T,
                                      int heads, int kvh, int hd, int vd, int page_size,
                                      int max_blocks, int window, float scale, float softcap,
                                      int keep_first, const float* sink, const void* gate,
                                      long long gate_ld, cudaStream_t stream) {
  return generic_checked(q, k_cache, v_cache, block_table, seq_of_token, positions, out, act_dtype,
                         T, heads, kvh, hd, vd, page_size, max_blocks, window, scale, softcap,
                         keep_first,
                         IxRows{(long long)heads * hd, (long long)heads * vd, 1.f, sink, gate,
                                gate_ld},
                         ix_no_distance(), stream);
}

// With a temperature and a distance penalty per head (see attention_distance.cuh).
IX_API int ix_distance_attention_generic(
    const void* q, long long q_ld, const void* k_cache, const void* v_cache,
    const int* block_table, const int* seq_of_token, const int* positions, void* out,
    long long o_ld, float o_scale, int act_dtype, int T, int heads, int kvh, int hd, int vd,
    int page_size, int max_blocks, float scale, const float* temp, const float* r1,
    const float* r2, int chunk, cudaStream_t stream) {
  if (!temp || !r1 || !r2 || chunk < 0) return IX_ERR_SIZE;
  return generic_checked(q, k_cache, v_cache, block_table, seq_of_token, positions, out, act_dtype,
                         T, heads, kvh, hd, vd, page_size, max_blocks, 0, scale, 0.f, 0,
                         IxRows{q_ld, o_ld, o_scale}, IxDistance{temp, r1, r2, chunk}, stream);
}
