// A residual made of several streams (hyper-connections).
//
// Per token the residual is S rows X_1 .. X_S of the model's width, float32, side by side ([tokens, S, width]).  A
// sublayer f with its norm n and its connection (a [S], B [S, S], c [S]) reads one combination of them and writes them all:
//
//     u = sum_s a_s X_s          y = f(n(u))          X'_t = sum_s B[s, t] X_s + c_t y          (all from the old X)
//
// with n(u) = u / sqrt(mean(u^2) + eps) * gain.  Everything is float32; only n(u), which the next product reads, leaves in
// the run's format.  Two kernels:
//
//  * streams_rows  - one block per row: the update with y (or none: only the combination), and the next sublayer's
//                    n(u) of the new streams (or none), so that a sublayer's end and the next one's beginning pass over
//                    the streams once.  Rows may be gathered by index when nothing is updated (the rows whose logits
//                    are wanted).
//  * streams_slices - the same for few tokens, a row spread over blocks of 256 columns: y arrives as the partial sums a
//                    product left (added in their order), and the next rows leave as u * gain without the norm's factor,
//                    beside each slice's sum of squares; whoever multiplies those rows applies the factor.
#include <type_traits>

#include "common.cuh"

namespace {

constexpr int MAX_STREAMS = 16;

// S > 0: that many streams, known when compiled; 0: `streams` of them, up to MAX_STREAMS.
template <int S>
struct Connection {
  static constexpr int CAP = S > 0 ? S : MAX_STREAMS;
};

// The new streams of one column from the old ones `x` and y: in place.
template <int S>
__device__ __forceinline__ void update_column(float (&x)[Connection<S>::CAP], int streams, const float* mix, const float* out, float y) {
  float old[Connection<S>::CAP];
#pragma unroll
  for (int s = 0; s < Connection<S>::CAP; ++s) old[s] = x[s];
#pragma unroll
  for (int t = 0; t < Connection<S>::CAP; ++t) {
    if (S == 0 && t >= streams) break;
    float v = out[t] * y;
#pragma unroll
    for (int s = 0; s < Connection<S>::CAP; ++s) {
      if (S == 0 && s >= streams) break;
      v = fmaf(mix[s * streams + t], old[s], v);
    }
    x[t] = v;
  }
}

template <int S>
__device__ __forceinline__ float combine_column(const float (&x)[Connection<S>::CAP], int streams, const float* in) {
  float u = 0.0f;
#pragma unroll
  for (int s = 0; s < Connection<S>::CAP; ++s) {
    if (S == 0 && s >= streams) break;
    u = fmaf(in[s], x[s], u);
  }
  return u;
}

// Threads of a block at most: the connection's numbers and four columns of every stream live in registers.
constexpr int block_limit(int streams) { return streams == 0 || streams > 4 ? 256 : 512; }

// Shared memory: [width] the row's u (when it is normed), then the connection's numbers.
template <int S, typename T, bool VEC>
__global__ void __launch_bounds__(block_limit(S)) streams_rows_kernel(
    float* __restrict__ x, int src_rows, int streams_arg, int width, const float* __restrict__ y, long long ld_y,
    const float* __restrict__ mix, const float* __restrict__ out, const float* __restrict__ in, const float* __restrict__ gain,
    float eps, const int* __restrict__ rows, T* __restrict__ h, int* status) {
  extern __shared__ __align__(16) float streams_smem[];
  __shared__ float scratch[32];
  __shared__ float c_mix[MAX_STREAMS * MAX_STREAMS], c_out[MAX_STREAMS], c_in[MAX_STREAMS];
  constexpr int CAP = Connection<S>::CAP;
  const int streams = S > 0 ? S : streams_arg;
  pdl_trigger();
  // the connection is the model's: it does not depend on the previous kernel
  if (y != nullptr) {
    for (int i = threadIdx.x; i < streams * streams; i += blockDim.x) c_mix[i] = mix[i];
    for (int i = threadIdx.x; i < streams; i += blockDim.x) c_out[i] = out[i];
  }
  if (h != nullptr)
    for (int i = threadIdx.x; i < streams; i += blockDim.x) c_in[i] = in != nullptr ? in[i] : 1.0f;
  pdl_wait();
  __syncthreads();
  const int r = blockIdx.x;
  const int src = rows != nullptr ? rows[r] : r;
  if (src < 0 || src >= src_rows) {
    if (threadIdx.x == 0) atomicOr(status, TGE_STATUS_BAD_ROW);
    return;
  }
  float* row = x + (size_t)src * streams * width;
  const float* yrow = y != nullptr ? y + (size_t)src * ld_y : nullptr;
  float sum = 0.0f;
  if (VEC) {
    for (int n = threadIdx.x * 4; n < width; n += blockDim.x * 4) {
      float v[4][CAP];
#pragma unroll
      for (int s = 0; s < CAP; ++s) {
        if (S == 0 && s >= streams) break;
        const float4 four = *reinterpret_cast<const float4*>(row + (size_t)s * width + n);
        v[0][s] = four.x; v[1][s] = four.y; v[2][s] = four.z; v[3][s] = four.w;
      }
      if (yrow != nullptr) {
        const float4 four = *reinterpret_cast<const float4*>(yrow + n);
        update_column<S>(v[0], streams, c_mix, c_out, four.x);
        update_column<S>(v[1], streams, c_mix, c_out, four.y);
        update_column<S>(v[2], streams, c_mix, c_out, four.z);
        update_column<S>(v[3], streams, c_mix, c_out, four.w);
#pragma unroll
        for (int s = 0; s < CAP; ++s) {
          if (S == 0 && s >= streams) break;
          *reinterpret_cast<float4*>(row + (size_t)s * width + n) = make_float4(v[0][s], v[1][s], v[2][s], v[3][s]);
        }
      }
      if (h != nullptr) {
        const float4 u = make_float4(combine_column<S>(v[0], streams, c_in), combine_column<S>(v[1], streams, c_in),
                                     combine_column<S>(v[2], streams, c_in), combine_column<S>(v[3], streams, c_in));
        *reinterpret_cast<float4*>(streams_smem + n) = u;
        sum = fmaf(u.x, u.x, sum); sum = fmaf(u.y, u.y, sum);
        sum = fmaf(u.z, u.z, sum); sum = fmaf(u.w, u.w, sum);
      }
    }
  } else {
    for (int n = threadIdx.x; n < width; n += blockDim.x) {
      float v[CAP];
#pragma unroll
      for (int s = 0; s < CAP; ++s) {
        if (S == 0 && s >= streams) break;
        v[s] = row[(size_t)s * width + n];
      }
      if (yrow != nullptr) {
        update_column<S>(v, streams, c_mix, c_out, yrow[n]);
#pragma unroll
        for (int s = 0; s < CAP; ++s) {
          if (S == 0 && s >= streams) break;
          row[(size_t)s * width + n] = v[s];
        }
      }
      if (h != nullptr) {
        const float u = combine_column<S>(v, streams, c_in);
        streams_smem[n] = u;
        sum = fmaf(u, u, sum);
      }
    }
  }
  if (h == nullptr) return;
  sum = block_sum(sum, scratch);
  const float scale = 1.0f / sqrtf(sum / (float)width + eps);
  T* dst = h + (size_t)r * width;
  if (VEC) {
    for (int n = threadIdx.x * 4; n < width; n += blockDim.x * 4) {       // every thread reads what it wrote
      const float4 u = *reinterpret_cast<const float4*>(streams_smem + n), g = *reinterpret_cast<const float4*>(gain + n);
      if (sizeof(T) == 2) {
        uint2 packed;
        *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(u.x * scale * g.x, u.y * scale * g.y);
        *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(u.z * scale * g.z, u.w * scale * g.w);
        *reinterpret_cast<uint2*>(dst + n) = packed;
      } else {
        *reinterpret_cast<float4*>(dst + n) = make_float4(u.x * scale * g.x, u.y * scale * g.y, u.z * scale * g.z, u.w * scale * g.w);
      }
    }
  } else {
    for (int n = threadIdx.x; n < width; n += blockDim.x) dst[n] = from_float<T>(streams_smem[n] * scale * gain[n]);
  }
}

constexpr int SLICE = 256;

// partial: float32 [splits, tokens, width] (null: nothing is updated).  scaled: bfloat16 [tokens, width] = u * gain; sums:
// float32 [slices, tokens], each slice's sum of u^2 (both null: only the update).
template <int S>
__global__ void __launch_bounds__(SLICE) streams_slices_kernel(float* __restrict__ x, int streams_arg, int width,
                                                               const float* __restrict__ partial, int splits, int tokens,
                                                               const float* __restrict__ mix, const float* __restrict__ out,
                                                               const float* __restrict__ in, const float* __restrict__ gain,
                                                               __nv_bfloat16* __restrict__ scaled, float* __restrict__ sums) {
  __shared__ float scratch[32];
  __shared__ float c_mix[MAX_STREAMS * MAX_STREAMS], c_out[MAX_STREAMS], c_in[MAX_STREAMS];
  constexpr int CAP = Connection<S>::CAP;
  const int streams = S > 0 ? S : streams_arg;
  pdl_trigger();
  const int t = blockIdx.y, n = blockIdx.x * SLICE + threadIdx.x;
  const bool inside = n < width;
  if (partial != nullptr) {
    for (int i = threadIdx.x; i < streams * streams; i += SLICE) c_mix[i] = mix[i];
    if (threadIdx.x < streams) c_out[threadIdx.x] = out[threadIdx.x];
  }
  if (scaled != nullptr && threadIdx.x < streams) c_in[threadIdx.x] = in != nullptr ? in[threadIdx.x] : 1.0f;
  const float g = (inside && scaled != nullptr) ? gain[n] : 0.0f;
  __syncthreads();
  pdl_wait();
  float u = 0.0f;
  if (inside) {
    float* row = x + (size_t)t * streams * width + n;
    float v[CAP];
#pragma unroll
    for (int s = 0; s < CAP; ++s) {
      if (S == 0 && s >= streams) break;
      v[s] = row[(size_t)s * width];
    }
    if (partial != nullptr) {
      const size_t plane = (size_t)tokens * width;
      const float* src = partial + (size_t)t * width + n;
      float y = 0.0f;
#pragma unroll 4
      for (int k = 0; k < splits; ++k) y += src[k * plane];
      update_column<S>(v, streams, c_mix, c_out, y);
#pragma unroll
      for (int s = 0; s < CAP; ++s) {
        if (S == 0 && s >= streams) break;
        row[(size_t)s * width] = v[s];
      }
    }
    if (scaled != nullptr) {
      u = combine_column<S>(v, streams, c_in);
      scaled[(size_t)t * width + n] = __float2bfloat16_rn(u * g);
    }
  }
  if (scaled == nullptr) return;
  const float sum = block_sum(u * u, scratch);
  if (threadIdx.x == 0) sums[(size_t)blockIdx.x * tokens + t] = sum;
}

template <typename F>
void with_streams(int streams, F&& run) {
  switch (streams) {
    case 1: run(std::integral_constant<int, 1>()); return;
    case 2: run(std::integral_constant<int, 2>()); return;
    case 3: run(std::integral_constant<int, 3>()); return;
    case 4: run(std::integral_constant<int, 4>()); return;
    case 6: run(std::integral_constant<int, 6>()); return;
    case 8: run(std::integral_constant<int, 8>()); return;
    default: run(std::integral_constant<int, 0>()); return;
  }
}

template <typename T>
int launch_rows(float* x, int rows_out, int src_rows, int streams, int width, const float* y, long long ld_y, const float* mix,
                const float* out, const float* in, const float* gain, float eps, const int* rows, T* h, int* status,
                cudaStream_t stream) {
  const bool vec = width % 4 == 0 && (y == nullptr || (ld_y % 4 == 0 && (uintptr_t)y % 16 == 0)) && (uintptr_t)x % 16 == 0 &&
                   (h == nullptr || ((uintptr_t)h % 16 == 0 && (uintptr_t)gain % 16 == 0));
  const size_t smem = h != nullptr ? (size_t)width * sizeof(float) : 0;
  TGE_REQUIRE(smem <= 200 * 1024, "residual streams: rows of %d do not fit shared memory", width);
  // few rows: a block as wide as the row; many: blocks of 256 threads, several on an SM
  const int places = vec ? (width + 3) / 4 : width;
  int threads = rows_out <= 2 * tge_sm_count() ? (places + 31) / 32 * 32 : 256;
  int rc = 0;
  with_streams(streams, [&](auto count) {
    constexpr int S = decltype(count)::value;
    const int block = threads < block_limit(S) ? threads : block_limit(S);
    auto run = [&](auto kernel) {
      if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
        tge_set_error("residual streams: cannot reserve %zu bytes of shared memory", smem);
        rc = -2;
        return;
      }
      tge_launch(kernel, dim3(rows_out), dim3(block), smem, stream, x, src_rows, streams, width, y, ld_y, mix, out, in, gain, eps,
                 rows, h, status);
    };
    if (vec && S != 0) run(streams_rows_kernel<S, T, S != 0>);
    else run(streams_rows_kernel<S, T, false>);
  });
  return rc != 0 ? rc : tge_launched("streams_rows", 1);
}

}  // namespace

// x float32 [src_rows, streams, width].  y (float32 [src_rows, width], row stride ld_y; null: none): the streams are updated in
// place with mix [streams, streams] and out [streams].  h (run dtype [rows_out, width]; null: none): the next sublayer's norm
// of the (new) streams' combination with in [streams] (null: all one), gain [width], eps.  rows (null: all rows in order)
// picks the rows to combine and goes without an update.
TGE_API int tge_streams_rows(float* x, int rows_out, int src_rows, int streams, int width, const float* y, long long ld_y,
                             const float* mix, const float* out, const float* in, const float* gain, float eps, const int* rows,
                             void* h, int is_bf16, int* status, cudaStream_t stream) {
  TGE_REQUIRE(rows_out >= 0 && src_rows >= 0 && streams > 0 && streams <= MAX_STREAMS && width > 0,
              "residual streams: %d streams (at most %d) of width %d", streams, MAX_STREAMS, width);
  TGE_REQUIRE(y == nullptr || (mix != nullptr && out != nullptr && ld_y >= width && rows == nullptr && rows_out == src_rows),
              "residual streams: an update needs its matrix and takes every row");
  TGE_REQUIRE(h == nullptr || (gain != nullptr && eps > 0.0f), "residual streams: a norm needs its weight and a positive eps");
  TGE_REQUIRE(y != nullptr || h != nullptr, "residual streams: nothing to do");
  if (rows_out == 0) return 0;
  if (is_bf16)
    return launch_rows<__nv_bfloat16>(x, rows_out, src_rows, streams, width, y, ld_y, mix, out, in, gain, eps, rows,
                                      (__nv_bfloat16*)h, status, stream);
  return launch_rows<float>(x, rows_out, src_rows, streams, width, y, ld_y, mix, out, in, gain, eps, rows, (float*)h, status, stream);
}

TGE_API int tge_streams_slices(int width) { return (width + SLICE - 1) / SLICE; }

// For few tokens.  partial: float32 [splits, tokens, width] (null: no update); scaled bf16 [tokens, width] and sums float32
// [tge_streams_slices(width), tokens] (both null: only the update).
TGE_API int tge_streams_update_defer(float* x, int tokens, int streams, int width, const float* partial, int splits, const float* mix,
                                     const float* out, const float* in, const float* gain, void* scaled, float* sums,
                                     cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && tokens <= 65535 && streams > 0 && streams <= MAX_STREAMS && width > 0,
              "residual streams: %d streams (at most %d) of width %d", streams, MAX_STREAMS, width);
  TGE_REQUIRE(partial == nullptr || (splits > 0 && mix != nullptr && out != nullptr), "residual streams: an update needs its matrix");
  TGE_REQUIRE((scaled == nullptr) == (sums == nullptr) && (scaled == nullptr || gain != nullptr), "residual streams: rows go with their sums");
  TGE_REQUIRE(partial != nullptr || scaled != nullptr, "residual streams: nothing to do");
  if (tokens == 0) return 0;
  with_streams(streams, [&](auto count) {
    constexpr int S = decltype(count)::value;
    tge_launch(streams_slices_kernel<S>, dim3((width + SLICE - 1) / SLICE, tokens), dim3(SLICE), 0, stream, x, streams, width,
               partial, splits, tokens, mix, out, in, gain, (__nv_bfloat16*)scaled, sums);
  });
  return tge_launched("streams_slices", 1);
}
