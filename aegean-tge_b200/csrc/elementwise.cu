// Embedding, RMSNorm, residual add, rotary rotation fused with the cache store.
//
// Formulas follow the reference's scalar kernels:
//   rms norm     src/cpu/scalar/norm_rope_scalar.cpp:8-21
//   rotate-half  src/cpu/scalar/norm_rope_scalar.cpp:23-41
//   cache write  src/models/qwen2.cpp:2308-2329 (rotated K and plain V, after the bias)
//   embedding    src/models/qwen2.cpp:1143-1152
#include "common.cuh"

// ---------------------------------------------------------------------------
// embedding: x[t, c, :] = table[ids[t], :] * scale as float32, for every copy c
// ---------------------------------------------------------------------------
template <typename T>
__global__ void embedding_kernel(const T* __restrict__ table, const int* __restrict__ ids,
                                 float* __restrict__ out, int hidden, int copies, int vocab, float scale, int* status) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int id = ids[t];
  float* dst = out + (size_t)t * copies * hidden;
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_TOKEN);
    for (int i = threadIdx.x; i < copies * hidden; i += blockDim.x) dst[i] = 0.0f;
    return;
  }
  const T* src = table + (size_t)id * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float v = to_float<T>(src[i]) * scale;
    for (int c = 0; c < copies; ++c) dst[(size_t)c * hidden + i] = v;
  }
}

TGE_API int tge_embedding(const void* table, int is_bf16, const int* ids, float* out, int tokens,
                          int hidden, int copies, int vocab, float scale, int* status, cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && hidden > 0 && copies > 0 && vocab > 0, "embedding: bad sizes tokens=%d hidden=%d copies=%d vocab=%d",
              tokens, hidden, copies, vocab);
  if (tokens == 0) return 0;
  if (is_bf16)
    tge_launch(embedding_kernel<__nv_bfloat16>, tokens, 256, 0, stream, (const __nv_bfloat16*)table, ids, out, hidden, copies, vocab, scale, status);
  else
    tge_launch(embedding_kernel<float>, tokens, 256, 0, stream, (const float*)table, ids, out, hidden, copies, vocab, scale, status);
  return tge_launched("embedding", 1);
}

// ---------------------------------------------------------------------------
// RMSNorm over the float32 stream; output in the run dtype.
//   s = sum x_i^2 ; scale = 1 / sqrt(s / dim + eps) ; out_i = x_i * scale * w_i
// One block per output row; optional row gather (rows[r] = source row).
// ---------------------------------------------------------------------------
template <typename TOut>
__global__ void rmsnorm_kernel(const float* __restrict__ x, const float* __restrict__ weight,
                               const int* __restrict__ rows, TOut* __restrict__ out, int hidden,
                               int src_rows, float eps, int* status) {
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  int src = rows ? rows[r] : r;
  if (src < 0 || src >= src_rows) {
    if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_ROW);
    src = 0;
  }
  const float* in = x + (size_t)src * hidden;
  float sum = 0.0f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float v = in[i];
    sum = fmaf(v, v, sum);
  }
  sum = block_sum(sum, scratch);
  const float scale = 1.0f / sqrtf(sum / (float)hidden + eps);
  TOut* dst = out + (size_t)r * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = from_float<TOut>(in[i] * scale * weight[i]);
}

// The same with 16-byte loads and the row held in registers between the two passes:
// hidden a multiple of 4 and at most 16 values per thread.
constexpr int NORM_VEC_ITERS = 4;

__device__ __forceinline__ void store4(float* dst, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store4(__nv_bfloat16* dst, float a, float b, float c, float d) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 packed;
  packed.x = *reinterpret_cast<const uint32_t*>(&lo);
  packed.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(dst) = packed;
}

template <typename TOut>
__global__ void __launch_bounds__(512) rmsnorm_vec_kernel(const float* __restrict__ x, const float* __restrict__ weight,
                                                          const int* __restrict__ rows, TOut* __restrict__ out,
                                                          int hidden, int src_rows, float eps, int* status) {
  __shared__ float scratch[32];
  pdl_trigger();
  const int quads = hidden >> 2;
  float4 gain[NORM_VEC_ITERS], value[NORM_VEC_ITERS];
#pragma unroll
  for (int k = 0; k < NORM_VEC_ITERS; ++k) {      // constants of the model: before the wait
    const int i = threadIdx.x + k * blockDim.x;
    gain[k] = i < quads ? reinterpret_cast<const float4*>(weight)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  const int r = blockIdx.x;
  int src = rows ? rows[r] : r;
  if (src < 0 || src >= src_rows) {
    if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_ROW);
    src = 0;
  }
  const float4* in = reinterpret_cast<const float4*>(x + (size_t)src * hidden);
  float sum = 0.0f;
#pragma unroll
  for (int k = 0; k < NORM_VEC_ITERS; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    value[k] = i < quads ? in[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    sum = fmaf(value[k].x, value[k].x, sum);
    sum = fmaf(value[k].y, value[k].y, sum);
    sum = fmaf(value[k].z, value[k].z, sum);
    sum = fmaf(value[k].w, value[k].w, sum);
  }
  sum = block_sum(sum, scratch);
  const float scale = 1.0f / sqrtf(sum / (float)hidden + eps);
  TOut* dst = out + (size_t)r * hidden;
#pragma unroll
  for (int k = 0; k < NORM_VEC_ITERS; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < quads)
      store4(dst + 4 * (size_t)i, value[k].x * scale * gain[k].x, value[k].y * scale * gain[k].y,
             value[k].z * scale * gain[k].z, value[k].w * scale * gain[k].w);
  }
}

TGE_API int tge_rmsnorm(const float* x, const float* weight, const int* rows, void* out, int out_is_bf16,
                        int out_rows, int src_rows, int hidden, float eps, int* status, cudaStream_t stream) {
  TGE_REQUIRE(out_rows >= 0 && hidden > 0 && src_rows >= 0, "rmsnorm: bad sizes rows=%d hidden=%d", out_rows, hidden);
  TGE_REQUIRE(eps > 0.0f, "rmsnorm: eps must be positive");
  if (out_rows == 0) return 0;
  int threads = hidden >= 2048 ? 512 : 256;
  const bool aligned = ((uintptr_t)x | (uintptr_t)weight | (uintptr_t)out) % 16 == 0;
  if (hidden % 4 == 0 && hidden / 4 <= NORM_VEC_ITERS * threads && aligned) {
    // more and smaller blocks per SM keep more loads in flight while others sit in their reduction
    if (hidden / 4 <= NORM_VEC_ITERS * 256) threads = 256;
    if (out_is_bf16)
      tge_launch(rmsnorm_vec_kernel<__nv_bfloat16>, out_rows, threads, 0, stream, x, weight, rows, (__nv_bfloat16*)out, hidden, src_rows, eps, status);
    else
      tge_launch(rmsnorm_vec_kernel<float>, out_rows, threads, 0, stream, x, weight, rows, (float*)out, hidden, src_rows, eps, status);
    return tge_launched("rmsnorm", 1);
  }
  if (out_is_bf16)
    tge_launch(rmsnorm_kernel<__nv_bfloat16>, out_rows, threads, 0, stream, x, weight, rows, (__nv_bfloat16*)out, hidden, src_rows, eps, status);
  else
    tge_launch(rmsnorm_kernel<float>, out_rows, threads, 0, stream, x, weight, rows, (float*)out, hidden, src_rows, eps, status);
  return tge_launched("rmsnorm", 1);
}

// ---------------------------------------------------------------------------
// x += y  (float32 stream, y in the run dtype)
// ---------------------------------------------------------------------------
template <typename T>
__global__ void add_to_stream_kernel(float* __restrict__ x, const T* __restrict__ y, size_t count, float alpha) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; i < count; i += stride) x[i] += alpha * to_float<T>(y[i]);
}

TGE_API int tge_add_to_stream(float* x, const void* y, int y_is_bf16, long long count, float alpha, cudaStream_t stream) {
  TGE_REQUIRE(count >= 0, "add_to_stream: negative count");
  if (count == 0) return 0;
  long long blocks = (count + 255) / 256;
  if (blocks > tge_sm_count() * 16) blocks = tge_sm_count() * 16;
  if (y_is_bf16)
    add_to_stream_kernel<__nv_bfloat16><<<(int)blocks, 256, 0, stream>>>(x, (const __nv_bfloat16*)y, (size_t)count, alpha);
  else
    add_to_stream_kernel<float><<<(int)blocks, 256, 0, stream>>>(x, (const float*)y, (size_t)count, alpha);
  return tge_launched("add_to_stream", 1);
}

// ---------------------------------------------------------------------------
// Rotary rotation of q and k (rotate-half pairing over the first `rotary`
// dimensions of each head) fused with the store of k and v into their pages.
//   lo' = lo*cos - hi*sin ; hi' = lo*sin + hi*cos      (float32)
// q is rotated in place inside the fused qkv rows; k is rotated on its way into
// the cache, v is copied.  A page is [kv_heads, page_size, head_dim].
// ---------------------------------------------------------------------------
template <typename T>
__global__ void rope_kv_store_kernel(T* __restrict__ qkv, int row_stride, const float* __restrict__ cos_table,
                                     const float* __restrict__ sin_table, int table_rows,
                                     const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                                     const int* __restrict__ block_table, int max_pages, T* __restrict__ k_pages,
                                     T* __restrict__ v_pages, int num_pages, int page_size, int heads, int kv_heads,
                                     int head_dim, int rotary, int store_kv, int* status) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int pos = positions[t];
  T* row = qkv + (size_t)t * row_stride;
  const int half = rotary / 2;
  const bool rotate = half > 0;
  if (rotate && (pos < 0 || pos >= table_rows)) {
    if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_ROW);
    return;
  }
  const float* cs = cos_table + (size_t)pos * half;
  const float* sn = sin_table + (size_t)pos * half;
  // queries, in place
  if (rotate) {
    for (int i = threadIdx.x; i < heads * half; i += blockDim.x) {
      const int h = i / half, d = i - h * half;
      T* v = row + (size_t)h * head_dim;
      const float lo = to_float<T>(v[d]), hi = to_float<T>(v[d + half]);
      const float c = cs[d], s = sn[d];
      v[d] = from_float<T>(lo * c - hi * s);
      v[d + half] = from_float<T>(lo * s + hi * c);
    }
  }
  if (!store_kv) return;
  const int seq = seq_of_token[t];
  const int page = block_table[(size_t)seq * max_pages + pos / page_size];
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_PAGE);
    return;
  }
  const int slot = pos % page_size;
  const T* k_row = row + (size_t)heads * head_dim;
  const T* v_row = k_row + (size_t)kv_heads * head_dim;
  for (int i = threadIdx.x; i < kv_heads * head_dim; i += blockDim.x) {
    const int h = i / head_dim, d = i - h * head_dim;
    const size_t dst = (((size_t)page * kv_heads + h) * page_size + slot) * head_dim + d;
    float kv;
    if (d < half) {
      const float lo = to_float<T>(k_row[i]), hi = to_float<T>(k_row[i + half]);
      kv = lo * cs[d] - hi * sn[d];
    } else if (d < rotary) {
      const float lo = to_float<T>(k_row[i - half]), hi = to_float<T>(k_row[i]);
      kv = lo * sn[d - half] + hi * cs[d - half];
    } else {
      kv = to_float<T>(k_row[i]);
    }
    k_pages[dst] = from_float<T>(kv);
    v_pages[dst] = v_row[i];
  }
}

// bfloat16 with everything a multiple of 8 elements: units of 16 bytes.  A unit is either a rotation
// (8 low and the 8 matching high elements of a q or k head) or a plain copy (v, and the tail of a k head
// beyond the rotary width).  Same formulas as above.
__device__ __forceinline__ void unpack8(const uint4& raw, float f[8]) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 v = __bfloat1622float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
}
__device__ __forceinline__ uint4 pack8(const float f[8]) {
  uint4 raw;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  return raw;
}

__global__ void rope_kv_store_vec_kernel(__nv_bfloat16* __restrict__ qkv, int row_stride, const float* __restrict__ cos_table,
                                         const float* __restrict__ sin_table, int table_rows,
                                         const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                                         const int* __restrict__ block_table, int max_pages,
                                         __nv_bfloat16* __restrict__ k_pages, __nv_bfloat16* __restrict__ v_pages,
                                         int num_pages, int page_size, int heads, int kv_heads, int head_dim, int rotary,
                                         int store_kv, int* status) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  __nv_bfloat16* row = qkv + (size_t)t * row_stride;
  const int half = rotary / 2;
  const int rot_units = half / 8, tail_units = (head_dim - rotary) / 8, dim_units = head_dim / 8;
  const int q_units = heads * rot_units;
  const int k_rot_units = store_kv ? kv_heads * rot_units : 0;
  const int k_tail_units = store_kv ? kv_heads * tail_units : 0;
  const int v_units = store_kv ? kv_heads * dim_units : 0;
  const int rotations = q_units + k_rot_units;
  const int total = rotations + k_tail_units + v_units;
  for (int u = threadIdx.x; u < total; u += blockDim.x) {
    // where the unit comes from depends on nothing that has to be looked up: ask for the data first,
    // then walk the chain position -> page
    int h, d;
    const __nv_bfloat16* src;
    __nv_bfloat16* page_base;      // k or v pages for units that go to the cache
    const bool rotation = u < rotations, is_q = u < q_units;
    if (rotation) {
      const int v = is_q ? u : u - q_units;
      h = v / rot_units; d = (v - h * rot_units) * 8;
      src = row + (size_t)(is_q ? h : heads + h) * head_dim + d;
      page_base = k_pages;
    } else if (u < rotations + k_tail_units) {
      const int v = u - rotations;
      h = v / tail_units; d = rotary + (v - h * tail_units) * 8;
      src = row + (size_t)(heads + h) * head_dim + d;
      page_base = k_pages;
    } else {
      const int v = u - rotations - k_tail_units;
      h = v / dim_units; d = (v - h * dim_units) * 8;
      src = row + (size_t)(heads + kv_heads + h) * head_dim + d;
      page_base = v_pages;
    }
    const uint4 first = *reinterpret_cast<const uint4*>(src);
    uint4 second = first;
    if (rotation) second = *reinterpret_cast<const uint4*>(src + half);
    const int pos = positions[t];
    if (rotation && (pos < 0 || pos >= table_rows)) {
      atomicOr(status, TGE_STATUS_BAD_ROW);
      continue;
    }
    __nv_bfloat16* dst = row + (size_t)h * head_dim + d;
    if (!is_q) {
      const int page = block_table[(size_t)seq_of_token[t] * max_pages + pos / page_size];
      if (page < 0 || page >= num_pages) {
        atomicOr(status, TGE_STATUS_BAD_PAGE);
        continue;
      }
      dst = page_base + (((size_t)page * kv_heads + h) * page_size + pos % page_size) * head_dim + d;
    }
    if (!rotation) {
      *reinterpret_cast<uint4*>(dst) = first;
      continue;
    }
    const float* cs = cos_table + (size_t)pos * half + d;
    const float* sn = sin_table + (size_t)pos * half + d;
    float lo[8], hi[8], c[8], s[8], out_lo[8], out_hi[8];
    *reinterpret_cast<float4*>(c) = *reinterpret_cast<const float4*>(cs);
    *reinterpret_cast<float4*>(c + 4) = *reinterpret_cast<const float4*>(cs + 4);
    *reinterpret_cast<float4*>(s) = *reinterpret_cast<const float4*>(sn);
    *reinterpret_cast<float4*>(s + 4) = *reinterpret_cast<const float4*>(sn + 4);
    unpack8(first, lo);
    unpack8(second, hi);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      out_lo[i] = lo[i] * c[i] - hi[i] * s[i];
      out_hi[i] = lo[i] * s[i] + hi[i] * c[i];
    }
    *reinterpret_cast<uint4*>(dst) = pack8(out_lo);
    *reinterpret_cast<uint4*>(dst + half) = pack8(out_hi);
  }
}

TGE_API int tge_rope_kv_store(void* qkv, int is_bf16, int row_stride, const float* cos_table, const float* sin_table,
                              int table_rows, const int* positions, const int* seq_of_token, const int* block_table,
                              int max_pages, void* k_pages, void* v_pages, int num_pages, int page_size, int tokens,
                              int heads, int kv_heads, int head_dim, int rotary, int store_kv, int* status,
                              cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && heads > 0 && kv_heads >= 0 && head_dim > 0, "rope_kv_store: bad sizes");
  TGE_REQUIRE(rotary >= 0 && rotary <= head_dim && rotary % 2 == 0,
              "rope_kv_store: rotary width %d must be even and at most head_dim %d", rotary, head_dim);
  TGE_REQUIRE(!store_kv || (page_size > 0 && max_pages > 0 && num_pages > 0), "rope_kv_store: bad page geometry");
  TGE_REQUIRE(row_stride >= (heads + (store_kv ? 2 * kv_heads : 0)) * head_dim, "rope_kv_store: row stride %d too small", row_stride);
  if (tokens == 0) return 0;
  const bool by_sixteen_bytes = is_bf16 && rotary % 16 == 0 && head_dim % 8 == 0 && row_stride % 8 == 0 &&
                                ((uintptr_t)qkv | (uintptr_t)cos_table | (uintptr_t)sin_table) % 16 == 0 &&
                                (!store_kv || ((uintptr_t)k_pages | (uintptr_t)v_pages) % 16 == 0);
  if (by_sixteen_bytes) {
    const int units = heads * (rotary / 16) + (store_kv ? kv_heads * (rotary / 16 + (head_dim - rotary) / 8 + head_dim / 8) : 0);
    int threads = (units + 31) / 32 * 32;
    if (threads > 512) threads = 512;
    if (threads < 32) threads = 32;
    tge_launch(rope_kv_store_vec_kernel, tokens, threads, 0, stream,
        (__nv_bfloat16*)qkv, row_stride, cos_table, sin_table, table_rows, positions, seq_of_token, block_table,
        max_pages, (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages, num_pages, page_size, heads, kv_heads, head_dim,
        rotary, store_kv, status);
    return tge_launched("rope_kv_store", 1);
  }
  if (is_bf16)
    tge_launch(rope_kv_store_kernel<__nv_bfloat16>, tokens, 256, 0, stream,
        (__nv_bfloat16*)qkv, row_stride, cos_table, sin_table, table_rows, positions, seq_of_token, block_table,
        max_pages, (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages, num_pages, page_size, heads, kv_heads, head_dim,
        rotary, store_kv, status);
  else
    tge_launch(rope_kv_store_kernel<float>, tokens, 256, 0, stream,
        (float*)qkv, row_stride, cos_table, sin_table, table_rows, positions, seq_of_token, block_table, max_pages,
        (float*)k_pages, (float*)v_pages, num_pages, page_size, heads, kv_heads, head_dim, rotary, store_kv, status);
  return tge_launched("rope_kv_store", 1);
}

// out[m, n] = rows[m, n] / sqrt(sum over slices of sums[slice][m] / width + eps), bfloat16: completes rows that
// travelled without their RMSNorm factor, for a taker that cannot apply it itself.
namespace {
__global__ void scale_rows_kernel(const __nv_bfloat16* __restrict__ rows, long long ld_rows, const float* __restrict__ sums,
                                  int slices, int width, float eps, __nv_bfloat16* __restrict__ out, long long ld_out,
                                  int m_rows, int n_cols) {
  pdl_trigger();
  pdl_wait();
  const int m = blockIdx.x;
  float sum = 0.0f;
  for (int slice = 0; slice < slices; ++slice) sum += sums[(size_t)slice * m_rows + m];
  const float factor = 1.0f / sqrtf(sum / (float)width + eps);
  for (int n = threadIdx.x; n < n_cols; n += blockDim.x)
    out[(size_t)m * ld_out + n] = __float2bfloat16_rn(__bfloat162float(rows[(size_t)m * ld_rows + n]) * factor);
}
}  // namespace

TGE_API int tge_scale_rows(const void* rows, long long ld_rows, const float* sums, int slices, int width, float eps,
                           void* out, long long ld_out, int m_rows, int n_cols, cudaStream_t stream) {
  TGE_REQUIRE(m_rows >= 0 && n_cols > 0 && slices > 0 && width > 0, "scale_rows: bad sizes");
  if (m_rows == 0) return 0;
  tge_launch(scale_rows_kernel, m_rows, 256, 0, stream, (const __nv_bfloat16*)rows, ld_rows, sums, slices, width, eps,
             (__nv_bfloat16*)out, ld_out, m_rows, n_cols);
  return tge_launched("scale_rows", 1);
}

// ---------------------------------------------------------------------------
// RMS norm of the query and key projections fused with a blend of the values and the cache store: what
// the rotate-and-store kernel is to a rotary layer, for a layer that normalises q and k instead.
//   q <- q / sqrt(mean(q^2) + eps) * wq      k <- k / sqrt(mean(k^2) + eps) * wk        (float32 statistics)
// The mean runs over the WHOLE projection of a token (all heads at once; weights of that size) or, with
// `per_head`, over each head by itself (weights of one head's size).  A null weight leaves that projection
// as it is.  With `v_other` the values become (1 - lambda) v + lambda v_other (lambda read from the device,
// v_other another layer's values of the same tokens); the blended values are what the pages get and what
// stays in the row.  q, k and v are rewritten in place inside the fused row [q | k | v]; k and v go to their
// pages, [kv_heads, page_size, head_dim] and [kv_heads, page_size, value_dim].  One block per token.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) qk_norm_kv_store_kernel(
    T* __restrict__ qkv, int row_stride, const float* __restrict__ q_weight, const float* __restrict__ k_weight,
    float eps, int per_head, const T* __restrict__ v_other, int v_other_stride, const float* __restrict__ blend,
    const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ block_table,
    int max_pages, T* __restrict__ k_pages, T* __restrict__ v_pages, int num_pages, int page_size, int heads,
    int kv_heads, int head_dim, int value_dim, int store_kv, int* status) {
  __shared__ float scratch[32];
  __shared__ float head_factor[256];
  pdl_trigger();
  const int t = blockIdx.x;
  const int pos = positions[t];
  const int seq = seq_of_token[t];
  const float lambda = blend != nullptr ? blend[0] : 0.0f;            // a model constant: not the previous kernel's work
  pdl_wait();
  T* row = qkv + (size_t)t * row_stride;
  T* k_row = row + (size_t)heads * head_dim;
  T* v_row = k_row + (size_t)kv_heads * head_dim;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;

  size_t k_base = 0, v_base = 0;
  bool store = store_kv != 0;
  if (store) {
    const int page_index = pos / page_size;
    const int page = (pos >= 0 && page_index < max_pages) ? block_table[(size_t)seq * max_pages + page_index] : -1;
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_PAGE);
      store = false;
    } else {
      k_base = ((size_t)page * kv_heads * page_size + (pos % page_size)) * head_dim;
      v_base = ((size_t)page * kv_heads * page_size + (pos % page_size)) * value_dim;
    }
  }

  // the two projections, one after the other: which == 0 queries, which == 1 keys
  for (int which = 0; which < 2; ++which) {
    T* base = which == 0 ? row : k_row;
    const float* weight = which == 0 ? q_weight : k_weight;
    const int count = (which == 0 ? heads : kv_heads);
    const int width = count * head_dim;
    if (weight != nullptr) {
      if (per_head) {
        for (int h0 = 0; h0 < count; h0 += 256) {
          for (int h = h0 + warp; h < min(count, h0 + 256); h += warps) {
            float sum = 0.0f;
            for (int d = lane; d < head_dim; d += 32) {
              const float v = to_float<T>(base[(size_t)h * head_dim + d]);
              sum = fmaf(v, v, sum);
            }
            sum = warp_sum(sum);
            if (lane == 0) head_factor[h - h0] = 1.0f / sqrtf(sum / (float)head_dim + eps);
          }
          __syncthreads();
          for (int i = h0 * head_dim + threadIdx.x; i < min(count, h0 + 256) * head_dim; i += blockDim.x) {
            const int h = i / head_dim;
            base[i] = from_float<T>(to_float<T>(base[i]) * head_factor[h - h0] * weight[i - h * head_dim]);
          }
          __syncthreads();
        }
      } else {
        float sum = 0.0f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) {
          const float v = to_float<T>(base[i]);
          sum = fmaf(v, v, sum);
        }
        const float factor = 1.0f / sqrtf(block_sum(sum, scratch) / (float)width + eps);
        for (int i = threadIdx.x; i < width; i += blockDim.x)
          base[i] = from_float<T>(to_float<T>(base[i]) * factor * weight[i]);
      }
    }
    if (which == 1 && store) {
      // every thread stores the elements it has just written itself
      const int step = (weight != nullptr && per_head) ? 0 : 1;
      if (step == 0) __syncthreads();
      for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const int h = i / head_dim, d = i - h * head_dim;
        k_pages[k_base + (size_t)h * page_size * head_dim + d] = k_row[i];
      }
    }
  }
  for (int i = threadIdx.x; i < kv_heads * value_dim; i += blockDim.x) {
    T v = v_row[i];
    if (v_other != nullptr) {
      const float mine = to_float<T>(v), other = to_float<T>(v_other[(size_t)t * v_other_stride + i]);
      v = from_float<T>((1.0f - lambda) * mine + lambda * other);
      v_row[i] = v;
    }
    if (store) {
      const int h = i / value_dim, d = i - h * value_dim;
      v_pages[v_base + (size_t)h * page_size * value_dim + d] = v;
    }
  }
}

// bfloat16 with every size a multiple of 8 elements and the norm over the whole projection: a token's row is read
// once in units of 16 bytes that stay in registers between the sums of squares and the scaling, so the row moves
// through memory once in and once out (and its k and v once more into the pages).
constexpr int QKN_THREADS = 256;
constexpr int QKN_UNITS = 12;          // most units per thread: rows of up to 256 * 12 * 8 = 24,576 elements

// UNITS: units of 16 bytes a thread holds (2, 4, 8 or 12, the least that covers the row: fewer registers, more
// blocks on an SM; with 12 for every row a 2,048-token step took 28 us where the rotate-and-store kernel takes 10).
template <int UNITS>
__global__ void __launch_bounds__(QKN_THREADS) qk_norm_kv_store_vec_kernel(
    __nv_bfloat16* __restrict__ qkv, int row_stride, const float* __restrict__ q_weight, const float* __restrict__ k_weight,
    float eps, const __nv_bfloat16* __restrict__ v_other, int v_other_stride, const float* __restrict__ blend,
    const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ block_table,
    int max_pages, __nv_bfloat16* __restrict__ k_pages, __nv_bfloat16* __restrict__ v_pages, int num_pages, int page_size,
    int heads, int kv_heads, int head_dim, int value_dim, int store_kv, int* status) {
  __shared__ float scratch[32];
  pdl_trigger();
  const int t = blockIdx.x;
  const int pos = positions[t];
  const float lambda = blend != nullptr ? blend[0] : 0.0f;
  bool store = store_kv != 0;
  size_t k_base = 0, v_base = 0;
  if (store) {
    const int page_index = pos / page_size;
    const int page = (pos >= 0 && page_index < max_pages) ? block_table[(size_t)seq_of_token[t] * max_pages + page_index] : -1;
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_PAGE);
      store = false;
    } else {
      k_base = ((size_t)page * kv_heads * page_size + (pos % page_size)) * head_dim;
      v_base = ((size_t)page * kv_heads * page_size + (pos % page_size)) * value_dim;
    }
  }
  pdl_wait();
  const int q_units = heads * head_dim / 8, k_units = kv_heads * head_dim / 8, v_units = kv_heads * value_dim / 8;
  const int units = q_units + k_units + v_units;
  uint4* row = reinterpret_cast<uint4*>(qkv + (size_t)t * row_stride);
  uint4 raw[UNITS];
#pragma unroll
  for (int i = 0; i < UNITS; ++i) {
    const int u = threadIdx.x + i * QKN_THREADS;
    raw[i] = u < units ? row[u] : make_uint4(0u, 0u, 0u, 0u);
  }
  float sum_q = 0.0f, sum_k = 0.0f;
#pragma unroll
  for (int i = 0; i < UNITS; ++i) {
    const int u = threadIdx.x + i * QKN_THREADS;
    if (u >= q_units + k_units) continue;
    float f[8];
    unpack8(raw[i], f);
    float part = 0.0f;
#pragma unroll
    for (int e = 0; e < 8; ++e) part = fmaf(f[e], f[e], part);
    if (u < q_units) sum_q += part; else sum_k += part;
  }
  {
    // both sums through one pair of barriers, in an order that depends on the block size alone
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    sum_q = warp_sum(sum_q);
    sum_k = warp_sum(sum_k);
    if (lane == 0) { scratch[warp] = sum_q; scratch[QKN_THREADS / 32 + warp] = sum_k; }
    __syncthreads();
    sum_q = warp_sum(lane < QKN_THREADS / 32 ? scratch[lane] : 0.0f);
    sum_k = warp_sum(lane < QKN_THREADS / 32 ? scratch[QKN_THREADS / 32 + lane] : 0.0f);
  }
  const float f_q = 1.0f / sqrtf(sum_q / (float)(q_units * 8) + eps);
  const float f_k = 1.0f / sqrtf(sum_k / (float)(k_units * 8) + eps);
#pragma unroll
  for (int i = 0; i < UNITS; ++i) {
    const int u = threadIdx.x + i * QKN_THREADS;
    if (u >= units) continue;
    float f[8];
    unpack8(raw[i], f);
    if (u < q_units + k_units) {
      const bool is_q = u < q_units;
      const float* weight = is_q ? q_weight : k_weight;
      if (weight != nullptr) {
        const float factor = is_q ? f_q : f_k;
        const int first = (is_q ? u : u - q_units) * 8;
        const float4 w0 = *reinterpret_cast<const float4*>(weight + first), w1 = *reinterpret_cast<const float4*>(weight + first + 4);
        f[0] *= factor * w0.x; f[1] *= factor * w0.y; f[2] *= factor * w0.z; f[3] *= factor * w0.w;
        f[4] *= factor * w1.x; f[5] *= factor * w1.y; f[6] *= factor * w1.z; f[7] *= factor * w1.w;
        raw[i] = pack8(f);
        row[u] = raw[i];
      }
      if (!is_q && store) {
        const int e0 = (u - q_units) * 8, h = e0 / head_dim, d = e0 - h * head_dim;
        *reinterpret_cast<uint4*>(k_pages + k_base + (size_t)h * page_size * head_dim + d) = raw[i];
      }
    } else {
      const int e0 = (u - q_units - k_units) * 8;
      if (v_other != nullptr) {
        float o[8];
        unpack8(*reinterpret_cast<const uint4*>(v_other + (size_t)t * v_other_stride + e0), o);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = (1.0f - lambda) * f[e] + lambda * o[e];
        raw[i] = pack8(f);
        row[u] = raw[i];
      }
      if (store) {
        const int h = e0 / value_dim, d = e0 - h * value_dim;
        *reinterpret_cast<uint4*>(v_pages + v_base + (size_t)h * page_size * value_dim + d) = raw[i];
      }
    }
  }
}

// The same for the norm over each head: `lanes` lanes (a power of two, one per 16 bytes of a head) share a head, which
// stays in registers between its sum of squares and its scaling.
__global__ void __launch_bounds__(QKN_THREADS) qk_head_norm_kv_store_vec_kernel(
    __nv_bfloat16* __restrict__ qkv, int row_stride, const float* __restrict__ q_weight, const float* __restrict__ k_weight,
    float eps, const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ block_table,
    int max_pages, __nv_bfloat16* __restrict__ k_pages, __nv_bfloat16* __restrict__ v_pages, int num_pages, int page_size,
    int heads, int kv_heads, int head_dim, int value_dim, int store_kv, int lanes, int* status) {
  pdl_trigger();
  const int t = blockIdx.x;
  const int pos = positions[t];
  bool store = store_kv != 0;
  size_t k_base = 0, v_base = 0;
  if (store) {
    const int page_index = pos / page_size;
    const int page = (pos >= 0 && page_index < max_pages) ? block_table[(size_t)seq_of_token[t] * max_pages + page_index] : -1;
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_PAGE);
      store = false;
    } else {
      k_base = ((size_t)page * kv_heads * page_size + (pos % page_size)) * head_dim;
      v_base = ((size_t)page * kv_heads * page_size + (pos % page_size)) * value_dim;
    }
  }
  pdl_wait();
  uint4* row = reinterpret_cast<uint4*>(qkv + (size_t)t * row_stride);
  const int per_head = head_dim / 8, total = heads + kv_heads;
  const int mine = threadIdx.x & (lanes - 1), groups = QKN_THREADS / lanes;
  for (int base = 0; base < total; base += groups) {
    const int unit = base + (int)threadIdx.x / lanes;
    const bool valid = unit < total && mine < per_head;
    const uint4 raw = valid ? row[unit * per_head + mine] : make_uint4(0u, 0u, 0u, 0u);
    float f[8];
    unpack8(raw, f);
    float sum = 0.0f;
#pragma unroll
    for (int e = 0; e < 8; ++e) sum = fmaf(f[e], f[e], sum);
    for (int step = lanes >> 1; step > 0; step >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, step);
    if (!valid) continue;                                  // the shuffles above were the last ones of this pass
    const bool is_q = unit < heads;
    const float* weight = is_q ? q_weight : k_weight;
    uint4 done = raw;
    if (weight != nullptr) {
      const float factor = 1.0f / sqrtf(sum / (float)head_dim + eps);
      const float4 w0 = *reinterpret_cast<const float4*>(weight + mine * 8), w1 = *reinterpret_cast<const float4*>(weight + mine * 8 + 4);
      f[0] *= factor * w0.x; f[1] *= factor * w0.y; f[2] *= factor * w0.z; f[3] *= factor * w0.w;
      f[4] *= factor * w1.x; f[5] *= factor * w1.y; f[6] *= factor * w1.z; f[7] *= factor * w1.w;
      done = pack8(f);
      row[unit * per_head + mine] = done;
    }
    if (!is_q && store)
      *reinterpret_cast<uint4*>(k_pages + k_base + (size_t)(unit - heads) * page_size * head_dim + mine * 8) = done;
  }
  if (!store) return;
  const uint4* v_row = row + total * per_head;
  for (int u = threadIdx.x; u < kv_heads * value_dim / 8; u += QKN_THREADS) {
    const int h = u * 8 / value_dim, d = u * 8 - h * value_dim;
    *reinterpret_cast<uint4*>(v_pages + v_base + (size_t)h * page_size * value_dim + d) = v_row[u];
  }
}

// qkv: [tokens, >= heads*head_dim + kv_heads*(head_dim + value_dim)] rows of [q | k | v], row stride in elements; no kv
// heads: rows of q alone (a layer that reads another layer's cache), nothing is stored.
// q_weight / k_weight: float32, heads*head_dim and kv_heads*head_dim long (or head_dim each with per_head), or null.
// v_other: null, or the other layer's values [tokens, kv_heads*value_dim] with its row stride; blend: device float.
TGE_API int tge_qk_norm_kv_store(void* qkv, int is_bf16, int row_stride, const float* q_weight, const float* k_weight,
                                 float eps, int per_head, const void* v_other, int v_other_stride, const float* blend,
                                 const int* positions, const int* seq_of_token, const int* block_table, int max_pages,
                                 void* k_pages, void* v_pages, int num_pages, int page_size, int tokens, int heads,
                                 int kv_heads, int head_dim, int value_dim, int store_kv, int* status,
                                 cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && heads > 0 && kv_heads >= 0 && head_dim > 0 && value_dim > 0, "qk_norm_kv_store: bad sizes");
  TGE_REQUIRE(kv_heads > 0 || !store_kv, "qk_norm_kv_store: without kv heads there is nothing to store");
  TGE_REQUIRE(row_stride >= heads * head_dim + kv_heads * (head_dim + value_dim), "qk_norm_kv_store: rows of %d elements "
              "do not hold q, k and v", row_stride);
  TGE_REQUIRE(eps > 0.0f || (q_weight == nullptr && k_weight == nullptr), "qk_norm_kv_store: eps must be positive");
  TGE_REQUIRE((v_other == nullptr) == (blend == nullptr), "qk_norm_kv_store: a blend needs both the other values and lambda");
  TGE_REQUIRE(!store_kv || (page_size > 0 && max_pages > 0 && num_pages > 0 && k_pages && v_pages && block_table),
              "qk_norm_kv_store: bad page geometry");
  if (tokens == 0) return 0;
  const bool aligned16 = ((uintptr_t)qkv % 16 == 0) && ((uintptr_t)v_other % 16 == 0) && ((uintptr_t)k_pages % 16 == 0) &&
                         ((uintptr_t)v_pages % 16 == 0) && ((uintptr_t)q_weight % 16 == 0) && ((uintptr_t)k_weight % 16 == 0);
  const long long units = ((long long)heads * head_dim + (long long)kv_heads * (head_dim + value_dim)) / 8;
  if (is_bf16 && !per_head && aligned16 && head_dim % 8 == 0 && value_dim % 8 == 0 && row_stride % 8 == 0 &&
      v_other_stride % 8 == 0 && units <= (long long)QKN_THREADS * QKN_UNITS) {
    const int per_thread = (int)((units + QKN_THREADS - 1) / QKN_THREADS);
    auto launch = [&](auto kernel) {
      tge_launch(kernel, tokens, QKN_THREADS, 0, stream, (__nv_bfloat16*)qkv, row_stride, q_weight, k_weight, eps,
                 (const __nv_bfloat16*)v_other, v_other_stride, blend, positions, seq_of_token, block_table, max_pages,
                 (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages, num_pages, page_size, heads, kv_heads, head_dim,
                 value_dim, store_kv, status);
    };
    if (per_thread <= 2) launch(qk_norm_kv_store_vec_kernel<2>);
    else if (per_thread <= 4) launch(qk_norm_kv_store_vec_kernel<4>);
    else if (per_thread <= 8) launch(qk_norm_kv_store_vec_kernel<8>);
    else launch(qk_norm_kv_store_vec_kernel<QKN_UNITS>);
    return tge_launched("qk_norm_kv_store_vec", 1);
  }
  if (is_bf16 && per_head && v_other == nullptr && aligned16 && head_dim % 8 == 0 && head_dim <= 256 && value_dim % 8 == 0 &&
      row_stride % 8 == 0) {
    int lanes = 1;
    while (lanes * 8 < head_dim) lanes *= 2;
    tge_launch(qk_head_norm_kv_store_vec_kernel, tokens, QKN_THREADS, 0, stream, (__nv_bfloat16*)qkv, row_stride, q_weight,
               k_weight, eps, positions, seq_of_token, block_table, max_pages, (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages,
               num_pages, page_size, heads, kv_heads, head_dim, value_dim, store_kv, lanes, status);
    return tge_launched("qk_head_norm_kv_store_vec", 1);
  }
  if (is_bf16)
    tge_launch(qk_norm_kv_store_kernel<__nv_bfloat16>, tokens, 256, 0, stream, (__nv_bfloat16*)qkv, row_stride, q_weight,
               k_weight, eps, per_head, (const __nv_bfloat16*)v_other, v_other_stride, blend, positions, seq_of_token,
               block_table, max_pages, (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages, num_pages, page_size, heads,
               kv_heads, head_dim, value_dim, store_kv, status);
  else
    tge_launch(qk_norm_kv_store_kernel<float>, tokens, 256, 0, stream, (float*)qkv, row_stride, q_weight, k_weight, eps,
               per_head, (const float*)v_other, v_other_stride, blend, positions, seq_of_token, block_table, max_pages,
               (float*)k_pages, (float*)v_pages, num_pages, page_size, heads, kv_heads, head_dim, value_dim, store_kv,
               status);
  return tge_launched("qk_norm_kv_store", 1);
}

// ---------------------------------------------------------------------------
// Soft cap of float32 scores, in place: z <- cap * tanh(z / cap).
// ---------------------------------------------------------------------------
__global__ void soft_cap_kernel(float* __restrict__ z, long long ld, int rows, int cols, float cap) {
  pdl_trigger();
  pdl_wait();
  const size_t count = (size_t)rows * cols;
  const float inv = 1.0f / cap;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / cols, c = i - r * cols;
    float* at = z + r * ld + c;
    *at = cap * tanhf(*at * inv);
  }
}

TGE_API int tge_soft_cap(float* z, long long ld, int rows, int cols, float cap, cudaStream_t stream) {
  TGE_REQUIRE(rows >= 0 && cols > 0 && ld >= cols && cap > 0.0f, "soft_cap: bad arguments");
  if (rows == 0) return 0;
  long long blocks = ((long long)rows * cols + 255) / 256;
  if (blocks > tge_sm_count() * 8) blocks = tge_sm_count() * 8;
  tge_launch(soft_cap_kernel, (int)blocks, 256, 0, stream, z, ld, rows, cols, cap);
  return tge_launched("soft_cap", 1);
}
