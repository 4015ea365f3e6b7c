// Memory-bound kernels of a step: embedding gather, residual-add + RMSNorm, SiLU-gate,
// rotary position encoding fused with the write of keys and values into cache pages.
// The residual stream is float32 in every precision mode; norm statistics and rotation
// are computed in float32.
#include "common.cuh"

// ---------------------------------------------------------------------------------
// Embedding: out[t, :] = table[ids[t], :]  (float32 residual stream), optionally plus pos_table[positions[t], :];
// `out2` (or null) receives the same rows once more (a model that keeps the embedding output beside the stream).
// ---------------------------------------------------------------------------------
template <typename TW>
__global__ void embed_gather_kernel(const TW* __restrict__ table, const int* __restrict__ ids,
                                    float* __restrict__ out, int H, int V, int* __restrict__ status, float scale,
                                    const TW* __restrict__ pos_table, const int* __restrict__ positions, int P,
                                    float* __restrict__ out2) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int t = blockIdx.x;
  const int id = ids[t];
  const int p = pos_table ? positions[t] : 0;
  if (id < 0 || id >= V || (pos_table && (p < 0 || p >= P))) {
    if (threadIdx.x == 0) atomicExch(status, 1);
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
      out[(size_t)t * H + j] = 0.f;
      if (out2) out2[(size_t)t * H + j] = 0.f;
    }
    return;
  }
  const TW* row = table + (size_t)id * H;
  if (pos_table || out2) {
    const TW* prow = pos_table ? pos_table + (size_t)p * H : nullptr;
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
      float x = co_to_float(row[j]);
      if (scale != 1.0f) x *= scale;
      if (prow) x += co_to_float(prow[j]);
      out[(size_t)t * H + j] = x;
      if (out2) out2[(size_t)t * H + j] = x;
    }
  } else if (scale == 1.0f) {
    for (int j = threadIdx.x; j < H; j += blockDim.x) out[(size_t)t * H + j] = co_to_float(row[j]);
  } else {   // an architecture that multiplies its embedding rows by a constant
    for (int j = threadIdx.x; j < H; j += blockDim.x) out[(size_t)t * H + j] = co_to_float(row[j]) * scale;
  }
}

// pos_table: [P][H] of the table's dtype, or null.
CO_EXPORT int coheryn_embed_gather(const void* table, int table_dtype, const int* ids, float* out,
                                   int T, int H, int V, int* status, float scale, const void* pos_table,
                                   const int* positions, int P, float* out2, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (pos_table && !positions) CO_FAIL("embed_gather: a row per position needs the positions");
  const int threads = H >= 1024 ? 256 : 128;
  if (table_dtype == CO_F32)
    co_launch(embed_gather_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)table, ids, out, H, V, status, scale,
              (const float*)pos_table, positions, P, out2);
  else if (table_dtype == CO_BF16)
    co_launch(embed_gather_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, (const __nv_bfloat16*)table, ids, out, H, V, status, scale,
              (const __nv_bfloat16*)pos_table, positions, P, out2);
  else
    CO_FAIL("embed_gather: unknown table dtype %d", table_dtype);
  CO_CHECK_LAUNCH("embed_gather");
  return 0;
}

// ---------------------------------------------------------------------------------
// Row gather: out[r, :] = src[rows[r], :] for rows of `row_bytes` bytes (any element type).
// ---------------------------------------------------------------------------------
template <typename Unit>
__global__ void gather_rows_kernel(const char* __restrict__ src, long src_stride, const int* __restrict__ rows,
                                   char* __restrict__ out, int units) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  const Unit* from = (const Unit*)(src + (size_t)rows[blockIdx.x] * src_stride);
  Unit* to = (Unit*)(out + (size_t)blockIdx.x * units * sizeof(Unit));
  for (int j = threadIdx.x; j < units; j += blockDim.x) to[j] = from[j];
}

CO_EXPORT int coheryn_gather_rows(const void* src, long src_stride_bytes, const int* rows, void* out, int R,
                                  int row_bytes, cudaStream_t stream) {
  if (R <= 0 || row_bytes <= 0) return 0;
  const bool wide = row_bytes % 16 == 0 && src_stride_bytes % 16 == 0 && ((uintptr_t)src % 16) == 0 && ((uintptr_t)out % 16) == 0;
  const bool words = row_bytes % 4 == 0 && src_stride_bytes % 4 == 0 && ((uintptr_t)src % 4) == 0 && ((uintptr_t)out % 4) == 0;
  if (wide)
    co_launch(gather_rows_kernel<uint4>, dim3(R), dim3(128), 0, stream, (const char*)src, src_stride_bytes, rows, (char*)out, row_bytes / 16);
  else if (words)
    co_launch(gather_rows_kernel<uint32_t>, dim3(R), dim3(128), 0, stream, (const char*)src, src_stride_bytes, rows, (char*)out, row_bytes / 4);
  else
    co_launch(gather_rows_kernel<unsigned char>, dim3(R), dim3(128), 0, stream, (const char*)src, src_stride_bytes, rows, (char*)out, row_bytes);
  CO_CHECK_LAUNCH("gather_rows");
  return 0;
}

// out[rows[r]] = src[r] for 32-bit elements (the inverse of a gather of single words).
__global__ void scatter_words_kernel(const uint32_t* __restrict__ src, const int* __restrict__ rows, uint32_t* __restrict__ out, int R) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.x * blockDim.x + threadIdx.x;
  if (r < R) out[rows[r]] = src[r];
}

CO_EXPORT int coheryn_scatter_words(const void* src, const int* rows, void* out, int R, cudaStream_t stream) {
  if (R <= 0) return 0;
  co_launch(scatter_words_kernel, dim3((R + 127) / 128), dim3(128), 0, stream, (const uint32_t*)src, rows, (uint32_t*)out, R);
  CO_CHECK_LAUNCH("scatter_words");
  return 0;
}

// ---------------------------------------------------------------------------------
// Logits of an architecture that scales them, adds a bias or caps them:
// x[r, v] = x[r, v] * scale + bias[v]; with cap > 0 then x = cap * tanh(x / cap).
// ---------------------------------------------------------------------------------
__global__ void scale_add_bias_kernel(float* __restrict__ x, long stride, int V, float scale, const void* __restrict__ bias,
                                      int bias_dtype, float cap) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  float* row = x + (size_t)blockIdx.y * stride;
  for (int v = blockIdx.x * blockDim.x + threadIdx.x; v < V; v += gridDim.x * blockDim.x) {
    float y = row[v] * scale + (bias ? co_load_any(bias, bias_dtype, v) : 0.f);
    if (cap > 0.f) y = cap * tanhf(y / cap);
    row[v] = y;
  }
}

CO_EXPORT int coheryn_scale_bias_cap(float* x, long stride, int R, int V, float scale, const void* bias, int bias_dtype,
                                     float cap, cudaStream_t stream) {
  if (R <= 0 || V <= 0) return 0;
  if (R > 65535) CO_FAIL("scale_add_bias: at most 65535 rows, not %d", R);
  const int blocks = (V + 1023) / 1024 < 64 ? (V + 1023) / 1024 : 64;
  co_launch(scale_add_bias_kernel, dim3(blocks, R), dim3(256), 0, stream, x, stride, V, scale, bias, bias_dtype, cap);
  CO_CHECK_LAUNCH("scale_add_bias");
  return 0;
}

CO_EXPORT int coheryn_scale_add_bias(float* x, long stride, int R, int V, float scale, const void* bias, int bias_dtype,
                                     cudaStream_t stream) {
  return coheryn_scale_bias_cap(x, stride, R, V, scale, bias, bias_dtype, 0.f, stream);
}

// ---------------------------------------------------------------------------------
// Something added to the float32 stream between two layers of the schedule (a model that runs a span of
// its layers several times adds its embedding again, and a vector per pass, before each pass):
// x[t, :] += table[ids[t], :] * scale (when a table is given) + vec[:] (when given).
// ---------------------------------------------------------------------------------
template <typename TW>
__global__ void stream_inject_kernel(float* __restrict__ x, const TW* __restrict__ table, const int* __restrict__ ids,
                                     float scale, const void* __restrict__ vec, int vec_dtype, int H, int V) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int t = blockIdx.x;
  const TW* row = nullptr;
  if (table) {
    const int id = ids[t];
    if (id >= 0 && id < V) row = table + (size_t)id * H;     // the embedding kernel has flagged an id outside the table
  }
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    float y = x[(size_t)t * H + j];
    if (row) y += co_to_float(row[j]) * scale;
    if (vec) y += co_load_any(vec, vec_dtype, j);
    x[(size_t)t * H + j] = y;
  }
}

CO_EXPORT int coheryn_stream_inject(float* x, const void* table, int table_dtype, const int* ids, float scale,
                                    const void* vec, int vec_dtype, int T, int H, int V, cudaStream_t stream) {
  if (T <= 0 || H <= 0 || (!table && !vec)) return 0;
  const int threads = H >= 1024 ? 256 : 128;
  if (table_dtype == CO_F32)
    co_launch(stream_inject_kernel<float>, dim3(T), dim3(threads), 0, stream, x, (const float*)table, ids, scale, vec, vec_dtype, H, V);
  else if (table_dtype == CO_BF16)
    co_launch(stream_inject_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, x, (const __nv_bfloat16*)table, ids, scale, vec,
              vec_dtype, H, V);
  else
    CO_FAIL("stream_inject: unknown table dtype %d", table_dtype);
  CO_CHECK_LAUNCH("stream_inject");
  return 0;
}

// ---------------------------------------------------------------------------------
// Residual add + RMSNorm.
//   x = resid[src] (+ delta[src]);  if update: resid[src] = x
//   out[r] = (x * (1/sqrt(mean(x^2) + eps))) * w
// src = rows ? rows[r] : r.  One block per row; the sum of squares is reduced in a
// fixed order, so a row's result does not depend on what else is in the batch.
// ---------------------------------------------------------------------------------
template <typename TD, typename TO>
__global__ void add_rmsnorm_kernel(float* __restrict__ resid, const TD* __restrict__ delta,
                                   const int* __restrict__ rows, const void* __restrict__ weight,
                                   int wdtype, float eps, TO* __restrict__ out, int H, int update) {
  __shared__ float scratch[33];
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.x;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* x = resid + src * H;
  const TD* d = delta ? delta + src * H : nullptr;
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    float v = x[j];
    if (d) {
      v += co_to_float(d[j]);
      if (update) x[j] = v;
    }
    ss += v * v;
  }
  ss = co_block_sum(ss, scratch);
  const float mean = ss / (float)H;
  const float scale = 1.0f / sqrtf(mean + eps);
  TO* o = out + (size_t)r * H;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    float v = x[j];
    if (d && !update) v += co_to_float(d[j]);
    o[j] = co_from_float<TO>((v * scale) * co_load_any(weight, wdtype, j));
  }
}

// Vector variant for widths that are a multiple of 4 and at most 8192: the row stays in
// registers between the two passes (float4 per thread and step), the delta is read four at
// a time.  Same arithmetic and the same order of summation per thread count.
template <typename T> struct Vec4;
template <> struct Vec4<float> {
  static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Vec4<__nv_bfloat16> {
  static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x);
    const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<unsigned*>(&a);
    raw.y = *reinterpret_cast<unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
  }
};

// Thread-block clusters: rank and size of this CTA's cluster (1 CTA when launched without one),
// and a sum over the cluster's CTAs: every CTA writes its term into slot `rank` of EVERY
// CTA's `slots` (distributed shared memory), the cluster meets at its hardware barrier, and
// each CTA adds its own copy of the slots in rank order.  No CTA reads a peer's memory, so
// none has to outlive the others.  `v` must be the same in all threads of the CTA.
__device__ __forceinline__ unsigned co_cluster_rank() { unsigned r; asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ unsigned co_cluster_size() { unsigned r; asm volatile("mov.u32 %0, %%cluster_nctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ float co_cluster_sum(float v, float* slots /* >= cluster size floats, shared */) {
  const unsigned n = co_cluster_size(), rank = co_cluster_rank();
  if (n == 1) return v;
  if (threadIdx.x < n) {
    unsigned local = (unsigned)__cvta_generic_to_shared(slots + rank), remote;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(threadIdx.x));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(v) : "memory");
  }
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
  float total = 0.f;
  for (unsigned k = 0; k < n; ++k) total += slots[k];
  return total;
}

template <typename TD, typename TO, typename TW, int STEPS>
__global__ void __launch_bounds__(256)
add_rmsnorm_vec_kernel(float* __restrict__ resid, const TD* __restrict__ delta, const int* __restrict__ rows,
                       const TW* __restrict__ weight, float eps, TO* __restrict__ out, int H, int update) {
  __shared__ float scratch[33];
  __shared__ float cl_slots[8];
  co_pdl_launch_dependents();
  // The CTAs of a cluster share a row: CTA k of n takes the k-th run of columns.
  const int cl_n = (int)co_cluster_size(), cl_r = (int)co_cluster_rank();
  const int c_per = ((H / 4 + cl_n - 1) / cl_n) * 4;
  const int c_lo = cl_r * c_per, c_hi = min(H, c_lo + c_per);
  float4 wv[STEPS];   // the weights depend on no earlier kernel
#pragma unroll
  for (int i = 0; i < STEPS; ++i) {
    const int j = c_lo + (i * 256 + threadIdx.x) * 4;
    wv[i] = j < c_hi ? Vec4<TW>::load(weight + j) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  co_pdl_wait();
  const int r = blockIdx.x / cl_n;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* x = resid + src * H;
  const TD* d = delta ? delta + src * H : nullptr;
  float4 v[STEPS];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < STEPS; ++i) {
    const int j = c_lo + (i * 256 + threadIdx.x) * 4;
    if (j < c_hi) {
      v[i] = Vec4<float>::load(x + j);
      if (d) {
        const float4 dv = Vec4<TD>::load(d + j);
        v[i].x += dv.x; v[i].y += dv.y; v[i].z += dv.z; v[i].w += dv.w;
        if (update) Vec4<float>::store(x + j, v[i]);
      }
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
  }
  ss = co_cluster_sum(co_block_sum(ss, scratch), cl_slots);
  const float scale = 1.0f / sqrtf(ss / (float)H + eps);
  TO* o = out + (size_t)r * H;
#pragma unroll
  for (int i = 0; i < STEPS; ++i) {
    const int j = c_lo + (i * 256 + threadIdx.x) * 4;
    if (j < c_hi) {
      const float4 w = wv[i];
      Vec4<TO>::store(o + j, make_float4((v[i].x * scale) * w.x, (v[i].y * scale) * w.y, (v[i].z * scale) * w.z,
                                         (v[i].w * scale) * w.w));
    }
  }
}

// Many rows (prompt portions): W warps per row (1, 2, 4 or 8: at most 16 float4 per lane), eight warps
// per CTA, so that a few hundred CTAs hold every row of the step at once, each row's loads are all
// in flight together and a one-warp row is reduced by shuffles alone.
template <typename TD, typename TO, typename TW, int VPL, int W>
__global__ void __launch_bounds__(256)
add_rmsnorm_rows_kernel(float* __restrict__ resid, const TD* __restrict__ delta, const int* __restrict__ rows,
                        const TW* __restrict__ weight, float eps, TO* __restrict__ out, int H, int update, int n_rows) {
  __shared__ float partial[8];
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.x * (8 / W) + warp / W, wsub = warp % W;
  const bool live = r < n_rows;
  const size_t src = live ? (rows ? (size_t)rows[r] : (size_t)r) : 0;
  float* x = resid + src * H;
  const TD* d = delta ? delta + src * H : nullptr;
  float4 v[VPL];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    const int j = ((i * W + wsub) * 32 + lane) * 4;
    v[i] = (live && j < H) ? Vec4<float>::load(x + j) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (d) {
    float4 dv[VPL];
#pragma unroll
    for (int i = 0; i < VPL; ++i) {
      const int j = ((i * W + wsub) * 32 + lane) * 4;
      dv[i] = (live && j < H) ? Vec4<TD>::load(d + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < VPL; ++i) {
      const int j = ((i * W + wsub) * 32 + lane) * 4;
      v[i].x += dv[i].x; v[i].y += dv[i].y; v[i].z += dv[i].z; v[i].w += dv[i].w;
      if (update && live && j < H) Vec4<float>::store(x + j, v[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < VPL; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  ss = co_warp_sum(ss);
  if (W > 1) {
    if (lane == 0) partial[warp] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < W; ++k) ss += partial[(warp / W) * W + k];
  }
  if (!live) return;
  const float scale = 1.0f / sqrtf(ss / (float)H + eps);
  TO* o = out + (size_t)r * H;
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    const int j = ((i * W + wsub) * 32 + lane) * 4;
    if (j < H) {
      const float4 w = Vec4<TW>::load(weight + j);
      Vec4<TO>::store(o + j, make_float4((v[i].x * scale) * w.x, (v[i].y * scale) * w.y, (v[i].z * scale) * w.z,
                                         (v[i].w * scale) * w.w));
    }
  }
}

// With few rows one CTA per row leaves the GPU idle and the row's latency long: a cluster of
// four CTAs shares each row (from 1024 columns on, up to 64 rows).
inline int norm_cluster(int n_rows, int H) { return (n_rows <= 64 && H >= 1024 && (H / 4) % 4 == 0) ? 4 : 1; }

template <typename TD, typename TO, typename TW>
void launch_rmsnorm_vec(float* resid, const void* delta, const int* rows, const void* weight, float eps, void* out,
                        int n_rows, int H, int update, cudaStream_t stream) {
  if (n_rows > 64) {
    // warps per row and float4 per lane: the fewest warps that keep a lane at 16 float4 or fewer
    int W = 1;
    while (W < 8 && (H / 4 + 32 * W - 1) / (32 * W) > 16) W *= 2;
    const int vpl = (H / 4 + 32 * W - 1) / (32 * W);
    const dim3 grid((n_rows + 8 / W - 1) / (8 / W));
#define ROWS(V, WW) co_launch(add_rmsnorm_rows_kernel<TD, TO, TW, V, WW>, grid, dim3(256), 0, stream, resid, (const TD*)delta, rows, \
                              (const TW*)weight, eps, (TO*)out, H, update, n_rows)
#define ROWS_W(WW) do { if (vpl <= 4) ROWS(4, WW); else if (vpl <= 8) ROWS(8, WW); else if (vpl <= 12) ROWS(12, WW); else ROWS(16, WW); } while (0)
    if (vpl <= 16) {
      if (W == 1) ROWS_W(1); else if (W == 2) ROWS_W(2); else if (W == 4) ROWS_W(4); else ROWS_W(8);
      return;
    }
#undef ROWS_W
#undef ROWS
  }
  const int cl = norm_cluster(n_rows, H);
  const int steps = (H / 4 / cl + 255) / 256;
#define GO(S) co_launch_cluster(cl, add_rmsnorm_vec_kernel<TD, TO, TW, S>, dim3(n_rows * cl), dim3(256), 0, stream, resid, \
                                (const TD*)delta, rows, (const TW*)weight, eps, (TO*)out, H, update)
  if (steps <= 1) GO(1); else if (steps <= 2) GO(2); else if (steps <= 4) GO(4); else GO(8);
#undef GO
}

CO_EXPORT int coheryn_add_rmsnorm(float* resid, const void* delta, int delta_dtype, const int* rows,
                                  const void* weight, int wdtype, float eps, void* out, int out_dtype,
                                  int n_rows, int H, int update, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (rows && update) CO_FAIL("add_rmsnorm: cannot update the residual through a row gather");
  if (H % 4 == 0 && H <= 8192 && ((uintptr_t)resid & 15) == 0 && ((uintptr_t)delta & 7) == 0 &&
      ((uintptr_t)weight & 15) == 0 && ((uintptr_t)out & 15) == 0 && (!delta || delta_dtype == out_dtype)) {
    const bool bf = out_dtype == CO_BF16;
    if (bf && wdtype == CO_BF16) launch_rmsnorm_vec<__nv_bfloat16, __nv_bfloat16, __nv_bfloat16>(resid, delta, rows, weight, eps, out, n_rows, H, update, stream);
    else if (bf) launch_rmsnorm_vec<__nv_bfloat16, __nv_bfloat16, float>(resid, delta, rows, weight, eps, out, n_rows, H, update, stream);
    else if (wdtype == CO_F32) launch_rmsnorm_vec<float, float, float>(resid, delta, rows, weight, eps, out, n_rows, H, update, stream);
    else launch_rmsnorm_vec<float, float, __nv_bfloat16>(resid, delta, rows, weight, eps, out, n_rows, H, update, stream);
    CO_CHECK_LAUNCH("add_rmsnorm");
    return 0;
  }
  const int threads = H >= 2048 ? 512 : (H >= 512 ? 256 : 128);
#define LAUNCH(TD, TO)                                                                              \
  co_launch(add_rmsnorm_kernel<TD, TO>, dim3(n_rows), dim3(threads), 0, stream, resid, (const TD*)delta, rows, \
            weight, wdtype, eps, (TO*)out, H, update)
  if (delta_dtype == CO_F32 && out_dtype == CO_F32) LAUNCH(float, float);
  else if (delta_dtype == CO_BF16 && out_dtype == CO_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
  else if (delta_dtype == CO_F32 && out_dtype == CO_BF16) LAUNCH(float, __nv_bfloat16);
  else if (delta_dtype == CO_BF16 && out_dtype == CO_F32) LAUNCH(__nv_bfloat16, float);
  else CO_FAIL("add_rmsnorm: unknown dtypes %d/%d", delta_dtype, out_dtype);
#undef LAUNCH
  CO_CHECK_LAUNCH("add_rmsnorm");
  return 0;
}

// The same with the delta given as a stack of float32 partial sums [splits][n][H] (a matrix
// product that split K over CTAs and left the addition to its consumer): the parts are added
// in order 0, 1, ... and then to the residual.  All of a thread's loads are independent.
template <typename TO, typename TW, int STEPS>
__global__ void __launch_bounds__(256)
add_parts_rmsnorm_vec_kernel(float* __restrict__ resid, const float* __restrict__ parts, int splits, size_t split_stride,
                             const int* __restrict__ rows, const TW* __restrict__ weight, float eps,
                             TO* __restrict__ out, int H, int update) {
  __shared__ float scratch[33];
  __shared__ float cl_slots[8];
  co_pdl_launch_dependents();
  // The CTAs of a cluster share a row: CTA k of n takes the k-th run of columns.
  const int cl_n = (int)co_cluster_size(), cl_r = (int)co_cluster_rank();
  const int c_per = ((H / 4 + cl_n - 1) / cl_n) * 4;
  const int c_lo = cl_r * c_per, c_hi = min(H, c_lo + c_per);
  float4 wv[STEPS];   // the weights depend on no earlier kernel
#pragma unroll
  for (int i = 0; i < STEPS; ++i) {
    const int j = c_lo + (i * 256 + threadIdx.x) * 4;
    wv[i] = j < c_hi ? Vec4<TW>::load(weight + j) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  co_pdl_wait();
  const int r = blockIdx.x / cl_n;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* x = resid + src * H;
  const float* d = parts + src * H;
  // Up to sixteen parts of every step are fetched before the first is added (the twelve heads of an
  // output projection, the twelve K slices of a down projection: one round trip); the additions
  // keep the order 0, 1, ...
  constexpr int ZB = STEPS == 1 ? 16 : 8;
  float4 v[STEPS], sum[STEPS];
#pragma unroll
  for (int i = 0; i < STEPS; ++i) {
    const int j = c_lo + (i * 256 + threadIdx.x) * 4;
    v[i] = j < c_hi ? Vec4<float>::load(x + j) : make_float4(0.f, 0.f, 0.f, 0.f);
    sum[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int z0 = 0; z0 < splits; z0 += ZB) {
    float4 t[STEPS][ZB];
#pragma unroll
    for (int i = 0; i < STEPS; ++i) {
      const int j = c_lo + (i * 256 + threadIdx.x) * 4;
#pragma unroll
      for (int u = 0; u < ZB; ++u)
        t[i][u] = (j < c_hi && z0 + u < splits) ? Vec4<float>::load(d + (size_t)(z0 + u) * split_stride + j)
                                             : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < STEPS; ++i)
#pragma unroll
      for (int u = 0; u < ZB; ++u) {
        sum[i].x += t[i][u].x; sum[i].y += t[i][u].y; sum[i].z += t[i][u].z; sum[i].w += t[i][u].w;
      }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < STEPS; ++i) {
    const int j = c_lo + (i * 256 + threadIdx.x) * 4;
    if (j < c_hi) {
      v[i].x += sum[i].x; v[i].y += sum[i].y; v[i].z += sum[i].z; v[i].w += sum[i].w;
      if (update) Vec4<float>::store(x + j, v[i]);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
  }
  ss = co_cluster_sum(co_block_sum(ss, scratch), cl_slots);
  const float scale = 1.0f / sqrtf(ss / (float)H + eps);
  TO* o = out + (size_t)r * H;
#pragma unroll
  for (int i = 0; i < STEPS; ++i) {
    const int j = c_lo + (i * 256 + threadIdx.x) * 4;
    if (j < c_hi) {
      const float4 w = wv[i];
      Vec4<TO>::store(o + j, make_float4((v[i].x * scale) * w.x, (v[i].y * scale) * w.y, (v[i].z * scale) * w.z,
                                         (v[i].w * scale) * w.w));
    }
  }
}

template <typename TO>
__global__ void add_parts_rmsnorm_kernel(float* __restrict__ resid, const float* __restrict__ parts, int splits,
                                         size_t split_stride, const int* __restrict__ rows,
                                         const void* __restrict__ weight, int wdtype, float eps, TO* __restrict__ out,
                                         int H, int update) {
  __shared__ float scratch[33];
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.x;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  float* x = resid + src * H;
  const float* d = parts + src * H;
  auto value = [&](int j) {
    float sum = d[j];
    for (int z = 1; z < splits; ++z) sum += d[z * split_stride + j];
    return x[j] + sum;
  };
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float v = value(j);
    ss += v * v;
  }
  ss = co_block_sum(ss, scratch);
  const float scale = 1.0f / sqrtf(ss / (float)H + eps);
  TO* o = out + (size_t)r * H;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float v = value(j);
    o[j] = co_from_float<TO>((v * scale) * co_load_any(weight, wdtype, j));
    if (update) x[j] = v;   // after the last read of x[j] by this thread, its only reader
  }
}

// parts: float32 [splits][n][H] with `split_stride` elements between splits (n = the rows of
// resid).  Otherwise as coheryn_add_rmsnorm.
CO_EXPORT int coheryn_add_parts_rmsnorm(float* resid, const float* parts, int splits, long split_stride,
                                        const int* rows, const void* weight, int wdtype, float eps, void* out,
                                        int out_dtype, int n_rows, int H, int update, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (splits < 1 || !parts) CO_FAIL("add_parts_rmsnorm: %d parts", splits);
  if (rows && update) CO_FAIL("add_parts_rmsnorm: cannot update the residual through a row gather");
  const bool bf = out_dtype == CO_BF16;
  if (!bf && out_dtype != CO_F32) CO_FAIL("add_parts_rmsnorm: unknown output dtype %d", out_dtype);
  if (H % 4 == 0 && H <= 8192 && (split_stride & 3) == 0 && ((uintptr_t)resid & 15) == 0 && ((uintptr_t)parts & 15) == 0 &&
      ((uintptr_t)weight & 15) == 0 && ((uintptr_t)out & 15) == 0) {
    const int cl = norm_cluster(n_rows, H);
    const int steps = (H / 4 / cl + 255) / 256;
#define GO2(TO, TW, S) co_launch_cluster(cl, add_parts_rmsnorm_vec_kernel<TO, TW, S>, dim3(n_rows * cl), dim3(256), 0, stream, resid, parts, \
                                 splits, (size_t)split_stride, rows, (const TW*)weight, eps, (TO*)out, H, update)
#define GO(TO, TW) do { if (steps <= 1) GO2(TO, TW, 1); else if (steps <= 2) GO2(TO, TW, 2); else if (steps <= 4) GO2(TO, TW, 4); else GO2(TO, TW, 8); } while (0)
    if (bf && wdtype == CO_BF16) GO(__nv_bfloat16, __nv_bfloat16);
    else if (bf) GO(__nv_bfloat16, float);
    else if (wdtype == CO_F32) GO(float, float);
    else GO(float, __nv_bfloat16);
#undef GO
#undef GO2
    CO_CHECK_LAUNCH("add_parts_rmsnorm");
    return 0;
  }
  const int threads = H >= 2048 ? 512 : (H >= 512 ? 256 : 128);
  if (bf) co_launch(add_parts_rmsnorm_kernel<__nv_bfloat16>, dim3(n_rows), dim3(threads), 0, stream, resid, parts, splits,
                    (size_t)split_stride, rows, weight, wdtype, eps, (__nv_bfloat16*)out, H, update);
  else co_launch(add_parts_rmsnorm_kernel<float>, dim3(n_rows), dim3(threads), 0, stream, resid, parts, splits,
                 (size_t)split_stride, rows, weight, wdtype, eps, (float*)out, H, update);
  CO_CHECK_LAUNCH("add_parts_rmsnorm");
  return 0;
}

// ---------------------------------------------------------------------------------
// Gated activation over interleaved columns: out[m, j] = silu(in[m, 2j]) * in[m, 2j+1],
// in is [M, 2I] (column 2j = gate_j, column 2j+1 = up_j).
// silu(g) = g / (1 + exp(-g)) in float32.
// ---------------------------------------------------------------------------------
template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ in, T* __restrict__ out, int I, size_t total, int code, float param,
                                long ldo) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total;
       i += (size_t)gridDim.x * blockDim.x) {
    const size_t m = i / I, j = i % I;
    float g = co_to_float(in[m * 2 * I + 2 * j]);
    float u = co_to_float(in[m * 2 * I + 2 * j + 1]);
    float r;
    if (code == CO_GATE_CLAMPED_SWISH) {     // the constant in full float32 here
      g = fminf(g, param);
      u = fminf(fmaxf(u, -param), param);
      r = g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
    } else {
      r = (code == 2 ? co_gelu_tanh(g) : g / (1.0f + expf(-g))) * u;
    }
    out[m * ldo + j] = co_from_float<T>(r);
  }
}

CO_EXPORT int coheryn_act_mul_ex(const void* in, void* out, int dtype, int M, int I, int code, float param, long ldo,
                                 cudaStream_t stream);
CO_EXPORT int coheryn_silu_mul(const void* in, void* out, int dtype, int M, int I, cudaStream_t stream) {
  return coheryn_act_mul_ex(in, out, dtype, M, I, 1, 0.f, I, stream);
}
CO_EXPORT int coheryn_act_mul(const void* in, void* out, int dtype, int M, int I, int code, cudaStream_t stream) {
  return coheryn_act_mul_ex(in, out, dtype, M, I, code, 0.f, I, stream);
}

// code: 1 SiLU, 2 the tanh form of GELU, 3 the clamped form with its constant `param` (the codes of the products' gated
// epilogues).  `ldo`: elements between the rows of out.
CO_EXPORT int coheryn_act_mul_ex(const void* in, void* out, int dtype, int M, int I, int code, float param, long ldo,
                                 cudaStream_t stream) {
  if (code < 1 || code > 3) CO_FAIL("act_mul: unknown activation code %d", code);
  if (code == 3 && !(param > 0.f)) CO_FAIL("act_mul: the clamp of activation 3 must be positive");
  const size_t total = (size_t)M * I;
  if (total == 0) return 0;
  const int threads = 256;
  const int blocks = (int)((total + threads - 1) / threads < 148 * 16 ? (total + threads - 1) / threads : 148 * 16);
  if (dtype == CO_F32) co_launch(silu_mul_kernel<float>, dim3(blocks), dim3(threads), 0, stream, (const float*)in, (float*)out, I, total, code, param, ldo);
  else if (dtype == CO_BF16) co_launch(silu_mul_kernel<__nv_bfloat16>, dim3(blocks), dim3(threads), 0, stream, (const __nv_bfloat16*)in, (__nv_bfloat16*)out, I, total, code, param, ldo);
  else CO_FAIL("silu_mul: unknown dtype %d", dtype);
  CO_CHECK_LAUNCH("silu_mul");
  return 0;
}

// ---------------------------------------------------------------------------------
// A residual add whose summand is normalised first, fused with the norm that reads the sum:
//   y = sum_p parts[p]                                     (inner == 0), or
//   y = coef * sum_p parts[p] / rms(parts[p]) * inner_w[p] (inner == 1: each part normalised by itself, a weight each)
//   x = resid + y / rms(y) * post_w;   resid = x (update);   out = x / rms(x) * w  (when w is given)
// rms(z) = sqrt(mean(z^2) + eps).  One CTA per row; the row's y and x live in shared memory ([2][H] floats).
// With `rows` the CTA r reads row rows[r] and the residual stays as it is.
// ---------------------------------------------------------------------------------
template <typename TO>
__global__ void __launch_bounds__(256)
add_normed_rmsnorm_kernel(float* __restrict__ resid, const float* __restrict__ parts, int n_parts, size_t part_stride, long ldp,
                          const void* __restrict__ inner_w, int inner_dtype, float coef, const void* __restrict__ post_w,
                          int post_dtype, const int* __restrict__ rows, const void* __restrict__ w, int w_dtype, float eps,
                          TO* __restrict__ out, int H, int update) {
  extern __shared__ __align__(16) float row_s[];
  __shared__ float scratch[33];
  float* ys = row_s;
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.x;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  const float invH = 1.0f / (float)H;
  for (int j = threadIdx.x; j < H; j += blockDim.x) ys[j] = 0.f;
  for (int p = 0; p < n_parts; ++p) {
    const float* d = parts + p * part_stride + src * ldp;
    float scale = 1.f;
    if (inner_w) {
      float ss = 0.f;
      for (int j = threadIdx.x; j < H; j += blockDim.x) ss = fmaf(d[j], d[j], ss);
      ss = co_block_sum(ss, scratch);
      scale = 1.0f / sqrtf(ss * invH + eps);
    }
    for (int j = threadIdx.x; j < H; j += blockDim.x)    // a thread touches its own elements of ys only
      ys[j] += inner_w ? (d[j] * scale) * co_load_any(inner_w, inner_dtype, (size_t)p * H + j) : d[j];
  }
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float y = inner_w ? ys[j] * coef : ys[j];
    ys[j] = y;
    ss = fmaf(y, y, ss);
  }
  ss = co_block_sum(ss, scratch);
  const float ps = 1.0f / sqrtf(ss * invH + eps);
  float* x = resid + src * H;
  float sx = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float v = x[j] + (ys[j] * ps) * co_load_any(post_w, post_dtype, j);
    ys[j] = v;
    if (update) x[j] = v;
    sx = fmaf(v, v, sx);
  }
  if (!w) return;
  sx = co_block_sum(sx, scratch);
  const float xs = 1.0f / sqrtf(sx * invH + eps);
  TO* o = out + (size_t)r * H;
  for (int j = threadIdx.x; j < H; j += blockDim.x) o[j] = co_from_float<TO>((ys[j] * xs) * co_load_any(w, w_dtype, j));
}

// Sums of N values over the CTA at once, the same in every thread (warp shuffles, then the warps' partials in order).
template <int N>
__device__ __forceinline__ void block_sum_n(float (&v)[N], float* scratch /* N * 32 floats, not in use by anyone else */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int n = 0; n < N; ++n) {
    v[n] = co_warp_sum(v[n]);
    if (lane == 0) scratch[n * 32 + warp] = v[n];
  }
  __syncthreads();
#pragma unroll
  for (int n = 0; n < N; ++n) {
    float t = 0.f;
    for (int w = 0; w < warps; ++w) t += scratch[n * 32 + w];
    v[n] = t;
  }
}

__device__ __forceinline__ float4 load4_any(const void* p, int dtype, size_t i4) {
  if (dtype == CO_F32) return reinterpret_cast<const float4*>(p)[i4];
  const uint2 raw = reinterpret_cast<const uint2*>(p)[i4];
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
  return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void store4(float* p, size_t i4, float4 v) { reinterpret_cast<float4*>(p)[i4] = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, size_t i4, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const unsigned*>(&a);
  raw.y = *reinterpret_cast<const unsigned*>(&b);
  reinterpret_cast<uint2*>(p)[i4] = raw;
}

// The same with the row in registers: H a multiple of 4 up to 1024 * VEC, every pointer on a 16-byte boundary, every
// global value read once by 16-byte loads, three reductions whatever the number of parts (at most two when each part is
// normalised by itself; any number when they are only added).
template <typename TO, int VEC>
__global__ void __launch_bounds__(256)
add_normed_rmsnorm_vec_kernel(float* __restrict__ resid, const float* __restrict__ parts, int n_parts, size_t part_stride, long ldp,
                              const void* __restrict__ inner_w, int inner_dtype, float coef, const void* __restrict__ post_w,
                              int post_dtype, const int* __restrict__ rows, const void* __restrict__ w, int w_dtype, float eps,
                              TO* __restrict__ out, int H, int update) {
  __shared__ float scratch[3][64];
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.x, H4 = H >> 2;
  const size_t src = rows ? (size_t)rows[r] : (size_t)r;
  const float invH = 1.0f / (float)H;
  float4 y[VEC];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  if (inner_w) {
    float4 d[2][VEC];
    float ss[2] = {0.f, 0.f};
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const int j = threadIdx.x + i * 256;
        d[p][i] = (p < n_parts && j < H4) ? reinterpret_cast<const float4*>(parts + p * part_stride + src * ldp)[j] : zero;
        ss[p] += d[p][i].x * d[p][i].x + d[p][i].y * d[p][i].y + d[p][i].z * d[p][i].z + d[p][i].w * d[p][i].w;
      }
    block_sum_n<2>(ss, scratch[0]);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int j = threadIdx.x + i * 256;
      y[i] = zero;
      if (j < H4)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          if (p >= n_parts) break;
          const float sc = 1.0f / sqrtf(ss[p] * invH + eps);
          const float4 wv = load4_any(inner_w, inner_dtype, (size_t)p * H4 + j);
          y[i].x += (d[p][i].x * sc) * wv.x; y[i].y += (d[p][i].y * sc) * wv.y;
          y[i].z += (d[p][i].z * sc) * wv.z; y[i].w += (d[p][i].w * sc) * wv.w;
        }
      y[i].x *= coef; y[i].y *= coef; y[i].z *= coef; y[i].w *= coef;
    }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const int j = threadIdx.x + i * 256;
      y[i] = zero;
      if (j < H4)
        for (int p = 0; p < n_parts; ++p) {
          const float4 dv = reinterpret_cast<const float4*>(parts + p * part_stride + src * ldp)[j];
          y[i].x += dv.x; y[i].y += dv.y; y[i].z += dv.z; y[i].w += dv.w;
        }
    }
  }
  float sy[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VEC; ++i) sy[0] += y[i].x * y[i].x + y[i].y * y[i].y + y[i].z * y[i].z + y[i].w * y[i].w;
  float* x = resid + src * H;
  // the stream and the weight of the summand's norm are requested before the reduction that their use waits for
  float4 xe[VEC], pe[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    xe[i] = j < H4 ? reinterpret_cast<const float4*>(x)[j] : zero;
    pe[i] = j < H4 ? load4_any(post_w, post_dtype, j) : zero;
  }
  block_sum_n<1>(sy, scratch[1]);
  const float ps = 1.0f / sqrtf(sy[0] * invH + eps);
  float sx[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    if (j < H4) {
      const float4 xv = xe[i], pw = pe[i];
      y[i] = make_float4(xv.x + (y[i].x * ps) * pw.x, xv.y + (y[i].y * ps) * pw.y, xv.z + (y[i].z * ps) * pw.z, xv.w + (y[i].w * ps) * pw.w);
      if (update) reinterpret_cast<float4*>(x)[j] = y[i];
      sx[0] += y[i].x * y[i].x + y[i].y * y[i].y + y[i].z * y[i].z + y[i].w * y[i].w;
    }
  }
  if (!w) return;
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    pe[i] = j < H4 ? load4_any(w, w_dtype, j) : zero;
  }
  block_sum_n<1>(sx, scratch[2]);
  const float xs = 1.0f / sqrtf(sx[0] * invH + eps);
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    if (j < H4) {
      const float4 wv = pe[i];
      store4(out + (size_t)r * H, (size_t)j, make_float4((y[i].x * xs) * wv.x, (y[i].y * xs) * wv.y, (y[i].z * xs) * wv.z, (y[i].w * xs) * wv.w));
    }
  }
}

// parts: float32 [n_parts][rows][H] (`part_stride` elements between parts, `ldp` between rows).  inner_w: [n_parts][H] or
// null.  w and out may be null: the residual is only updated.
CO_EXPORT int coheryn_add_normed_rmsnorm(float* resid, const float* parts, int n_parts, long part_stride, long ldp,
                                         const void* inner_w, int inner_dtype, float coef, const void* post_w, int post_dtype,
                                         const int* rows, const void* w, int w_dtype, float eps, void* out, int out_dtype,
                                         int n_rows, int H, int update, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (n_parts < 1 || !parts || !post_w) CO_FAIL("add_normed_rmsnorm: %d parts", n_parts);
  if (rows && update) CO_FAIL("add_normed_rmsnorm: cannot update the residual through a row gather");
  if ((w == nullptr) != (out == nullptr)) CO_FAIL("add_normed_rmsnorm: a weight and an output go together");
  const auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (H % 4 == 0 && H <= 8192 && (part_stride & 3) == 0 && (ldp & 3) == 0 && aligned(resid) && aligned(parts) && aligned(inner_w) &&
      aligned(post_w) && aligned(w) && aligned(out) && (!inner_w || n_parts <= 2) && (out_dtype == CO_BF16 || out_dtype == CO_F32)) {
    const int steps = (H / 4 + 255) / 256;
#define GO2(TO, V) co_launch(add_normed_rmsnorm_vec_kernel<TO, V>, dim3(n_rows), dim3(256), 0, stream, resid, parts, n_parts, \
                             (size_t)part_stride, ldp, inner_w, inner_dtype, coef, post_w, post_dtype, rows, w, w_dtype, eps, (TO*)out, H, update)
#define GO(TO) do { if (steps <= 1) GO2(TO, 1); else if (steps <= 2) GO2(TO, 2); else if (steps <= 4) GO2(TO, 4); else GO2(TO, 8); } while (0)
    if (out_dtype == CO_BF16) GO(__nv_bfloat16); else GO(float);
#undef GO
#undef GO2
    CO_CHECK_LAUNCH("add_normed_rmsnorm");
    return 0;
  }
  const size_t smem = (size_t)H * sizeof(float);
  const int threads = H >= 1024 ? 256 : 128;
  if (out_dtype == CO_BF16) {
    auto kern = add_normed_rmsnorm_kernel<__nv_bfloat16>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    co_launch(kern, dim3(n_rows), dim3(threads), smem, stream, resid, parts, n_parts, (size_t)part_stride, ldp, inner_w,
              inner_dtype, coef, post_w, post_dtype, rows, w, w_dtype, eps, (__nv_bfloat16*)out, H, update);
  } else if (out_dtype == CO_F32) {
    auto kern = add_normed_rmsnorm_kernel<float>;
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    co_launch(kern, dim3(n_rows), dim3(threads), smem, stream, resid, parts, n_parts, (size_t)part_stride, ldp, inner_w,
              inner_dtype, coef, post_w, post_dtype, rows, w, w_dtype, eps, (float*)out, H, update);
  } else {
    CO_FAIL("add_normed_rmsnorm: unknown output dtype %d", out_dtype);
  }
  CO_CHECK_LAUNCH("add_normed_rmsnorm");
  return 0;
}

// ---------------------------------------------------------------------------------
// A residual add followed by an average over depth, fused with the norm that reads the average:
//   y = sum_p parts[p];  x = resid + y / rms(y) * post_w   (post_w given), or x = resid + y   (no parts: x = resid)
//   s = sum_{j < n} avg_w[j] * hist[j] + avg_w[n] * x       (hist[j]: what the stream was after j earlier layers)
//   hist[n] = x (when keep);  resid = s (when update);  out = s / rms(s) * w  (when w is given)
// rms(z) = sqrt(mean(z^2) + eps).  One CTA per row.  With `rows` the CTA r reads row rows[r] of the stream, the parts and
// the history and nothing is written but `out`; `hist_rows` names the history's rows when they are not the stream's.
// ---------------------------------------------------------------------------------
struct DepthArgs {
  float* resid;
  const float* parts; int n_parts; size_t part_stride; long ldp;
  const void* post_w; int post_dtype;
  float* hist; size_t hist_stride; const float* avg_w; int n;
  const int* rows; const int* hist_rows;
  const void* w; int w_dtype; float eps;
  int H, update, keep;
};

template <typename TO>
__global__ void __launch_bounds__(256) depth_average_norm_kernel(DepthArgs A, TO* __restrict__ out) {
  extern __shared__ __align__(16) float row_s[];
  __shared__ float scratch[33];
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.x, H = A.H;
  const size_t src = A.rows ? (size_t)A.rows[r] : (size_t)r;
  const size_t hrow = A.hist_rows ? (size_t)A.hist_rows[src] : src;
  const float invH = 1.0f / (float)H;
  float ss = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {       // a thread touches its own elements of the row only
    float y = 0.f;
    for (int p = 0; p < A.n_parts; ++p) y += A.parts[p * A.part_stride + src * A.ldp + j];
    row_s[j] = y;
    ss = fmaf(y, y, ss);
  }
  float ps = 1.f;
  if (A.post_w) {
    ss = co_block_sum(ss, scratch);
    ps = 1.0f / sqrtf(ss * invH + A.eps);
  }
  float* x = A.resid + src * H;
  const float wn = A.avg_w[A.n];
  float sx = 0.f;
  for (int j = threadIdx.x; j < H; j += blockDim.x) {
    const float y = row_s[j];
    const float v = x[j] + (A.post_w ? (y * ps) * co_load_any(A.post_w, A.post_dtype, j) : y);
    float s = 0.f;
    for (int k = 0; k < A.n; ++k) s = fmaf(A.avg_w[k], A.hist[k * A.hist_stride + hrow * H + j], s);
    s = fmaf(wn, v, s);
    if (A.keep) A.hist[A.n * A.hist_stride + hrow * H + j] = v;
    if (A.update) x[j] = s;
    row_s[j] = s;
    sx = fmaf(s, s, sx);
  }
  if (!A.w) return;
  sx = co_block_sum(sx, scratch);
  const float xs = 1.0f / sqrtf(sx * invH + A.eps);
  TO* o = out + (size_t)r * H;
  for (int j = threadIdx.x; j < H; j += blockDim.x) o[j] = co_from_float<TO>((row_s[j] * xs) * co_load_any(A.w, A.w_dtype, j));
}

// The same with the row in registers (H a multiple of 4 up to 1024 * VEC, everything on 16-byte boundaries): the history
// is requested and summed before the reduction over the summand that the rest waits for.
template <typename TO, int VEC>
__global__ void __launch_bounds__(256) depth_average_norm_vec_kernel(DepthArgs A, TO* __restrict__ out) {
  __shared__ float scratch[2][32];
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int r = blockIdx.x, H = A.H, H4 = H >> 2;
  const size_t src = A.rows ? (size_t)A.rows[r] : (size_t)r;
  const size_t hrow = A.hist_rows ? (size_t)A.hist_rows[src] : src;
  const float invH = 1.0f / (float)H;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 y[VEC], s[VEC];
  float* x = A.resid + src * H;
  float sy[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    y[i] = zero;
    if (j < H4)
      for (int p = 0; p < A.n_parts; ++p) {
        const float4 d = reinterpret_cast<const float4*>(A.parts + p * A.part_stride + src * A.ldp)[j];
        y[i].x += d.x; y[i].y += d.y; y[i].z += d.z; y[i].w += d.w;
      }
    sy[0] += y[i].x * y[i].x + y[i].y * y[i].y + y[i].z * y[i].z + y[i].w * y[i].w;
  }
  float4 xe[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    xe[i] = j < H4 ? reinterpret_cast<const float4*>(x)[j] : zero;
    s[i] = zero;
    if (j < H4) {
#pragma unroll 8
      for (int k = 0; k < A.n; ++k) {
        const float wk = A.avg_w[k];
        const float4 h = reinterpret_cast<const float4*>(A.hist + k * A.hist_stride + hrow * H)[j];
        s[i].x = fmaf(wk, h.x, s[i].x); s[i].y = fmaf(wk, h.y, s[i].y); s[i].z = fmaf(wk, h.z, s[i].z); s[i].w = fmaf(wk, h.w, s[i].w);
      }
    }
  }
  float ps = 1.f;
  if (A.post_w) {
    block_sum_n<1>(sy, scratch[0]);
    ps = 1.0f / sqrtf(sy[0] * invH + A.eps);
  }
  const float wn = A.avg_w[A.n];
  float sx[1] = {0.f};
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    if (j < H4) {
      float4 v = y[i];
      if (A.post_w) {
        const float4 pw = load4_any(A.post_w, A.post_dtype, j);
        v = make_float4((v.x * ps) * pw.x, (v.y * ps) * pw.y, (v.z * ps) * pw.z, (v.w * ps) * pw.w);
      }
      v = make_float4(xe[i].x + v.x, xe[i].y + v.y, xe[i].z + v.z, xe[i].w + v.w);
      if (A.keep) reinterpret_cast<float4*>(A.hist + A.n * A.hist_stride + hrow * H)[j] = v;
      s[i] = make_float4(fmaf(wn, v.x, s[i].x), fmaf(wn, v.y, s[i].y), fmaf(wn, v.z, s[i].z), fmaf(wn, v.w, s[i].w));
      if (A.update) reinterpret_cast<float4*>(x)[j] = s[i];
      sx[0] += s[i].x * s[i].x + s[i].y * s[i].y + s[i].z * s[i].z + s[i].w * s[i].w;
    }
  }
  if (!A.w) return;
  block_sum_n<1>(sx, scratch[1]);
  const float xs = 1.0f / sqrtf(sx[0] * invH + A.eps);
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int j = threadIdx.x + i * 256;
    if (j < H4) {
      const float4 wv = load4_any(A.w, A.w_dtype, j);
      store4(out + (size_t)r * H, (size_t)j, make_float4((s[i].x * xs) * wv.x, (s[i].y * xs) * wv.y, (s[i].z * xs) * wv.z, (s[i].w * xs) * wv.w));
    }
  }
}

// hist: float32 [> n][history rows][H] (`hist_stride` elements between results); avg_w: float32 [n + 1].  parts, post_w, w
// and out may be null.
CO_EXPORT int coheryn_depth_average_norm(float* resid, const float* parts, int n_parts, long part_stride, long ldp,
                                         const void* post_w, int post_dtype, float* hist, long hist_stride, const float* avg_w,
                                         int n, const int* rows, const int* hist_rows, const void* w, int w_dtype, float eps,
                                         void* out, int out_dtype, int n_rows, int H, int update, int keep, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (n < 1 || !hist || !avg_w) CO_FAIL("depth_average_norm: an average needs its history");
  if ((parts == nullptr) != (n_parts == 0) || (post_w && !parts)) CO_FAIL("depth_average_norm: %d parts", n_parts);
  if ((rows && update) || ((rows || hist_rows) && keep)) CO_FAIL("depth_average_norm: cannot write through a row gather");
  if ((w == nullptr) != (out == nullptr)) CO_FAIL("depth_average_norm: a weight and an output go together");
  if (out && out_dtype != CO_F32 && out_dtype != CO_BF16) CO_FAIL("depth_average_norm: unknown output dtype %d", out_dtype);
  const DepthArgs A{resid, parts, n_parts, (size_t)part_stride, ldp, post_w, post_dtype, hist, (size_t)hist_stride, avg_w, n,
                    rows, hist_rows, w, w_dtype, eps, H, update, keep};
  const bool bf = out && out_dtype == CO_BF16;
  const auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (H % 4 == 0 && H <= 8192 && (part_stride & 3) == 0 && (ldp & 3) == 0 && (hist_stride & 3) == 0 && aligned(resid) &&
      aligned(parts) && aligned(post_w) && aligned(hist) && aligned(w) && aligned(out)) {
    const int steps = (H / 4 + 255) / 256;
#define GO2(TO, V) co_launch(depth_average_norm_vec_kernel<TO, V>, dim3(n_rows), dim3(256), 0, stream, A, (TO*)out)
#define GO(TO) do { if (steps <= 1) GO2(TO, 1); else if (steps <= 2) GO2(TO, 2); else if (steps <= 4) GO2(TO, 4); else GO2(TO, 8); } while (0)
    if (bf) GO(__nv_bfloat16); else GO(float);
#undef GO
#undef GO2
  } else {
    const size_t smem = (size_t)H * sizeof(float);
    const int threads = H >= 1024 ? 256 : 128;
#define GO(TO)                                                                                                              \
  do {                                                                                                                      \
    auto kern = depth_average_norm_kernel<TO>;                                                                              \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);               \
    co_launch(kern, dim3(n_rows), dim3(threads), smem, stream, A, (TO*)out);                                                \
  } while (0)
    if (bf) GO(__nv_bfloat16); else GO(float);
#undef GO
  }
  CO_CHECK_LAUNCH("depth_average_norm");
  return 0;
}

// ---------------------------------------------------------------------------------
// Rotary position encoding (rotate-half pairing (i, i + rot/2)) of q and k, fused with
// the write of k and v into their cache pages.
//   qkv: [T, (nh + 2 nkv) * hd]; q is rotated in place; rotated k and plain v go to
//   k_cache / v_cache, laid out [page][kv head][slot in page][hd].
//   cos_sin: float2 [max_pos][rot/2] = (cos, sin) of the angle of pair i at a position.
//   slots[t] = page * page_size + offset, or < 0 to write nothing for token t.
// Rotation is done in float32: out_a = fma(a, cos, -(b sin)), out_b = fma(a, sin, b cos).
// ---------------------------------------------------------------------------------
template <typename T>
__global__ void rope_kv_write_kernel(T* __restrict__ qkv, const int* __restrict__ positions,
                                     const float2* __restrict__ cos_sin, const int* __restrict__ slots,
                                     T* __restrict__ k_cache, T* __restrict__ v_cache, int nh, int nkv,
                                     int hd, int rot, int page_size, int write_kv) {
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int t = blockIdx.x;
  const int head = blockIdx.y;  // [0, nh): q   [nh, nh+nkv): k   [nh+nkv, nh+2nkv): v
  const int row_stride = (nh + 2 * nkv) * hd;
  T* src = qkv + (size_t)t * row_stride + (size_t)head * hd;
  const int pos = positions[t];
  const int half = rot >> 1;
  T* dst = nullptr;
  if (head >= nh) {
    if (!write_kv) return;
    const int slot = slots[t];
    if (slot < 0) return;
    const int page = slot / page_size, off = slot % page_size;
    const int kvh = head < nh + nkv ? head - nh : head - nh - nkv;
    T* base = head < nh + nkv ? k_cache : v_cache;
    dst = base + (((size_t)page * nkv + kvh) * page_size + off) * hd;
  }
  if (head < nh + nkv) {
    const float2* cs = cos_sin + (size_t)pos * half;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      const float a = co_to_float(src[i]), b = co_to_float(src[i + half]);
      const float2 c = cs[i];
      const T ra = co_from_float<T>(fmaf(a, c.x, -(b * c.y)));
      const T rb = co_from_float<T>(fmaf(a, c.y, b * c.x));
      if (dst) { dst[i] = ra; dst[i + half] = rb; }
      else { src[i] = ra; src[i + half] = rb; }
    }
    if (dst)
      for (int i = rot + threadIdx.x; i < hd; i += blockDim.x) dst[i] = src[i];
  } else {
    for (int i = threadIdx.x; i < hd; i += blockDim.x) dst[i] = src[i];
  }
}

// Vector variant: one block per token; an item is 16 bytes of a head's first half together
// with the matching 16 bytes of its second half (q and k heads), or 16 bytes of a v head.
// Needs rot == hd and hd/2 a multiple of the vector width.
template <typename T>
__global__ void __launch_bounds__(128)
rope_kv_write_vec_kernel(T* __restrict__ qkv, const int* __restrict__ positions, const float2* __restrict__ cos_sin,
                         const int* __restrict__ slots, T* __restrict__ k_cache, T* __restrict__ v_cache, int nh,
                         int nkv, int hd, int page_size, int write_kv) {
  constexpr int VEC = 16 / sizeof(T);
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int t = blockIdx.x;
  const int half = hd >> 1, per_half = half / VEC, per_head = hd / VEC;
  T* row = qkv + (size_t)t * (nh + 2 * nkv) * hd;
  const int pos = positions[t];
  const float2* cs = cos_sin + (size_t)pos * half;
  const int slot = write_kv ? slots[t] : -1;
  const int page = slot >= 0 ? slot / page_size : 0, off = slot >= 0 ? slot % page_size : 0;
  const int rot_items = (nh + (write_kv ? nkv : 0)) * per_half;
  const int items = rot_items + (write_kv ? nkv * per_head : 0);
  for (int it = threadIdx.x; it < items; it += blockDim.x) {
    if (it < rot_items) {
      const int head = it / per_half, c = (it % per_half) * VEC;
      T* src = row + (size_t)head * hd;
      T a[VEC], b[VEC];
      *reinterpret_cast<uint4*>(a) = *reinterpret_cast<const uint4*>(src + c);
      *reinterpret_cast<uint4*>(b) = *reinterpret_cast<const uint4*>(src + half + c);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float fa = co_to_float(a[i]), fb = co_to_float(b[i]);
        const float2 k = cs[c + i];
        a[i] = co_from_float<T>(fmaf(fa, k.x, -(fb * k.y)));
        b[i] = co_from_float<T>(fmaf(fa, k.y, fb * k.x));
      }
      T* dst = src;
      if (head >= nh) {
        if (slot < 0) continue;
        dst = k_cache + (((size_t)page * nkv + (head - nh)) * page_size + off) * hd;
      }
      *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(a);
      *reinterpret_cast<uint4*>(dst + half + c) = *reinterpret_cast<const uint4*>(b);
    } else {
      if (slot < 0) continue;
      const int j = it - rot_items;
      const int kvh = j / per_head, c = (j % per_head) * VEC;
      const T* src = row + (size_t)(nh + nkv + kvh) * hd;
      T* dst = v_cache + (((size_t)page * nkv + kvh) * page_size + off) * hd;
      *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(src + c);
    }
  }
}

// The same for a q/k/v product whose K slices have not been added yet: value(t, col) = sum over
// the slices of parts[s][t][col] (in order, from zero) + bias[col], rounded to bfloat16 as the
// product's own output would be, then rotated; q goes to q_out [T, nh * hd], k and v to the cache.
__global__ void __launch_bounds__(32)
rope_kv_write_parts_kernel(const float* __restrict__ parts, int splits, size_t split_stride, const void* __restrict__ bias,
                           int bias_dtype, __nv_bfloat16* __restrict__ q_out, const int* __restrict__ positions,
                           const float2* __restrict__ cos_sin, const int* __restrict__ slots,
                           __nv_bfloat16* __restrict__ k_cache, __nv_bfloat16* __restrict__ v_cache, int nh, int nkv, int hd,
                           int page_size) {
  typedef __nv_bfloat16 T;
  constexpr int VEC = 8;
  co_pdl_launch_dependents();
  co_pdl_wait();
  const int t = blockIdx.x;
  const int half = hd >> 1, per_half = half / VEC, per_head = hd / VEC;
  const size_t width = (size_t)(nh + 2 * nkv) * hd;
  const float* row = parts + (size_t)t * width;
  const int pos = positions[t];
  const float2* cs = cos_sin + (size_t)pos * half;
  const int slot = slots[t];
  const int page = slot >= 0 ? slot / page_size : 0, off = slot >= 0 ? slot % page_size : 0;
  auto gather = [&](size_t col, float (&v)[VEC]) {      // eight columns from col, slices added in order, bias, rounding
    float4 lo = make_float4(0.f, 0.f, 0.f, 0.f), hi = lo;
    for (int z = 0; z < splits; ++z) {
      const float4 a = *reinterpret_cast<const float4*>(row + (size_t)z * split_stride + col);
      const float4 b = *reinterpret_cast<const float4*>(row + (size_t)z * split_stride + col + 4);
      lo.x += a.x; lo.y += a.y; lo.z += a.z; lo.w += a.w;
      hi.x += b.x; hi.y += b.y; hi.z += b.z; hi.w += b.w;
    }
    v[0] = lo.x; v[1] = lo.y; v[2] = lo.z; v[3] = lo.w; v[4] = hi.x; v[5] = hi.y; v[6] = hi.z; v[7] = hi.w;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      if (bias) v[i] += co_load_any(bias, bias_dtype, col + i);
      v[i] = __bfloat162float(__float2bfloat16_rn(v[i]));
    }
  };
  // One block per (token, head): heads 0 .. nh - 1 are queries, then the keys, then the values.
  const int head = blockIdx.y;
  if (head < nh + nkv) {
    for (int it = threadIdx.x; it < per_half; it += blockDim.x) {
      const int c = it * VEC;
      float fa[VEC], fb[VEC];
      gather((size_t)head * hd + c, fa);
      gather((size_t)head * hd + half + c, fb);
      T a[VEC], b[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const float2 k = cs[c + i];
        a[i] = __float2bfloat16_rn(fmaf(fa[i], k.x, -(fb[i] * k.y)));
        b[i] = __float2bfloat16_rn(fmaf(fa[i], k.y, fb[i] * k.x));
      }
      T* dst;
      if (head < nh) dst = q_out + ((size_t)t * nh + head) * hd;
      else {
        if (slot < 0) continue;
        dst = k_cache + (((size_t)page * nkv + (head - nh)) * page_size + off) * hd;
      }
      *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(a);
      *reinterpret_cast<uint4*>(dst + half + c) = *reinterpret_cast<const uint4*>(b);
    }
  } else if (slot >= 0) {
    const int kvh = head - nh - nkv;
    for (int it = threadIdx.x; it < per_head; it += blockDim.x) {
      const int c = it * VEC;
      float fv[VEC];
      gather((size_t)head * hd + c, fv);
      T v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = __float2bfloat16_rn(fv[i]);
      T* dst = v_cache + (((size_t)page * nkv + kvh) * page_size + off) * hd;
      *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(v);
    }
  }
}

// parts: float32 [splits][T][(nh + 2 nkv) * hd]; the whole head is rotated (rotary size = hd, hd / 2 a
// multiple of 8); q_out: bfloat16 [T, nh * hd].
CO_EXPORT int coheryn_rope_kv_write_parts(const float* parts, int splits, long split_stride, const void* bias, int bias_dtype,
                                          void* q_out, const int* positions, const float* cos_sin, const int* slots,
                                          void* k_cache, void* v_cache, int T, int nh, int nkv, int hd, int page_size,
                                          cudaStream_t stream) {
  if (T <= 0) return 0;
  if (splits < 1 || (hd / 2) % 8 || (hd & 1)) CO_FAIL("rope_kv_write_parts: %d parts, head size %d", splits, hd);
  if (((uintptr_t)parts & 15) || (split_stride & 3) || ((uintptr_t)q_out & 15) || ((uintptr_t)k_cache & 15) || ((uintptr_t)v_cache & 15))
    CO_FAIL("rope_kv_write_parts: operands must be 16-byte aligned");
  if (nh + 2 * nkv > 65535) CO_FAIL("rope_kv_write_parts: %d heads", nh + 2 * nkv);
  co_launch(rope_kv_write_parts_kernel, dim3(T, nh + 2 * nkv), dim3(32), 0, stream, parts, splits, (size_t)split_stride, bias, bias_dtype,
            (__nv_bfloat16*)q_out, positions, (const float2*)cos_sin, slots, (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, nh,
            nkv, hd, page_size);
  CO_CHECK_LAUNCH("rope_kv_write_parts");
  return 0;
}

CO_EXPORT int coheryn_rope_kv_write(void* qkv, int dtype, const int* positions, const float* cos_sin,
                                    const int* slots, void* k_cache, void* v_cache, int T, int nh, int nkv,
                                    int hd, int rot, int page_size, int write_kv, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot < 0 || rot > hd || (rot & 1)) CO_FAIL("rope_kv_write: rotary size %d does not fit head size %d", rot, hd);
  const int vec = dtype == CO_F32 ? 4 : 8;
  if (rot == hd && (hd / 2) % vec == 0 && ((uintptr_t)qkv & 15) == 0 && ((uintptr_t)k_cache & 15) == 0 &&
      ((uintptr_t)v_cache & 15) == 0) {
    if (dtype == CO_F32)
      co_launch(rope_kv_write_vec_kernel<float>, dim3(T), dim3(128), 0, stream, (float*)qkv, positions,
                (const float2*)cos_sin, slots, (float*)k_cache, (float*)v_cache, nh, nkv, hd, page_size, write_kv);
    else if (dtype == CO_BF16)
      co_launch(rope_kv_write_vec_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, stream, (__nv_bfloat16*)qkv, positions,
                (const float2*)cos_sin, slots, (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, nh, nkv, hd, page_size,
                write_kv);
    else CO_FAIL("rope_kv_write: unknown dtype %d", dtype);
    CO_CHECK_LAUNCH("rope_kv_write");
    return 0;
  }
  dim3 grid(T, nh + 2 * nkv);
  const int threads = hd >= 128 ? 64 : 32;
  if (dtype == CO_F32)
    co_launch(rope_kv_write_kernel<float>, grid, dim3(threads), 0, stream, (float*)qkv, positions, (const float2*)cos_sin, slots,
              (float*)k_cache, (float*)v_cache, nh, nkv, hd, rot, page_size, write_kv);
  else if (dtype == CO_BF16)
    co_launch(rope_kv_write_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, (__nv_bfloat16*)qkv, positions, (const float2*)cos_sin, slots,
              (__nv_bfloat16*)k_cache, (__nv_bfloat16*)v_cache, nh, nkv, hd, rot, page_size, write_kv);
  else CO_FAIL("rope_kv_write: unknown dtype %d", dtype);
  CO_CHECK_LAUNCH("rope_kv_write");
  return 0;
}
