// The matrix memory of an mLSTM mixer: per head a matrix S [dim, vdim], a normaliser n [dim] and a running maximum m,
// all float32 in a per-request slot, with a log input gate i and a log forget gate f per token:
//
//    i = cap tanh(zi / cap)      f = logsigmoid(cap tanh(zf / cap))
//    m' = max(f + m, i)          S' = exp(f + m - m') S + exp(i - m') k v^T        n' likewise with k alone
//    o  = S'^T q / (max(|n' . q|, exp(-m')) + 1e-6)
//    y  = o / rms(o) * w * sigmoid(g)                              (the readout's norm per head and its gate)
//
//  * mlstm_step - token by token, a block per (head, request): S stays in registers over the request's tokens of the
//                 step, and the readout is normalised, weighted and gated before it is written, so a single token
//                 costs one read and one write of its state and nothing else;
//  * mlstm_gate_scan, mlstm_chunk_write, mlstm_chunk_carry, mlstm_chunk_read - portions of many tokens, in chunks of 64.
//                 With F_t the running sum of f over the portion, g_t = i_t - F_t and M_t = m_t - F_t (the running maximum
//                 of the g and of the m the portion starts with), a token s reaches a later token t with the factor
//                 exp(g_s - M_t) and the state from before a chunk with exp(M_before - M_t): so a chunk's own contribution to
//                 the state and the readout of a chunk are products. The scan works F, g and M out (float64: F grows with the
//                 portion), one kernel forms every chunk's own contribution, one carries the state from chunk to chunk, one
//                 reads out, normalises, weights and gates. The products run on the tensor cores with one operand in
//                 bfloat16 as it came from the projections and the other, a float32 number (a factor, a factor times a key,
//                 an entry of the state), as the sum of three bfloat16 numbers, which hold its 24 bits; accumulation is
//                 float32.
//
// Gates, the maximum, the normaliser, the state and the readout are float32 in both number formats; q, k, v and g come
// from a product in the run's format.
#include "common.cuh"

namespace {

constexpr float DENOMINATOR_FLOOR = 1e-6f;

__device__ __forceinline__ float sigmoid_m(float z) { return 1.0f / (1.0f + expf(-z)); }
// for an output gate whose product is rounded to bfloat16
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
__device__ __forceinline__ float log_sigmoid_m(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap_m(float z, float cap) { return cap * tanhf(z / cap); }

struct MlstmParams {
  const void* rows;            // [tokens, ld]: q (heads x dim), k, v (heads x vdim), g
  long long ld;
  const float* gates;          // [tokens, ld_gates]: zi (heads), zf (heads), their biases in them
  long long ld_gates;
  const float* norm_w;         // [heads * vdim]
  float* state;                // [slots, heads, dim, vdim]
  float* normaliser;           // [slots, heads, dim]
  float* maximum;              // [slots, heads]
  const int* slots;
  const int* q_start;
  void* out;                   // [tokens, ldo]
  long long ldo;
  int heads, dim, vdim, longest;
  float cap, q_scale, eps;
};

// R: rows of the state a thread holds (four columns each) in registers; 0: the state stays in memory (large heads).
// Thread (rg, cq) owns columns 4 cq .. 4 cq + 3 of rows rg, rg + RG, ...  Portions of more than `longest` tokens are
// left to another kernel.
template <typename T, int R>
__global__ void mlstm_step_kernel(const MlstmParams p) {
  extern __shared__ __align__(16) float step_smem[];
  __shared__ float scratch[32];
  pdl_trigger();
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int first = p.q_start[seq], last = p.q_start[seq + 1];
  const int slot = p.slots[seq];
  pdl_wait();                                  // before the return: no grid may finish ahead of the kernel before it
  if (first >= last || last - first > p.longest) return;
  const int dim = p.dim, vdim = p.vdim;
  const int quads = (vdim + 3) / 4, row_groups = blockDim.x / quads;
  const int cq = tid % quads, rg = tid / quads;
  const bool active = rg < row_groups;
  const bool vec = (vdim & 3) == 0;
  const int padded = (dim + 3) & ~3;           // every array below starts on 16 bytes
  float* qs = step_smem;                       // [dim]
  float* ks = qs + padded;                     // [dim]
  float* ns = ks + padded;                     // [dim]
  float* vs = ns + padded;                     // [4 quads]
  float* os = vs + 4 * quads;                  // [4 quads]
  float* part = os + 4 * quads;                // [row_groups][4 quads]
  const size_t unit = (size_t)slot * p.heads + head;
  float* S = p.state + unit * dim * vdim;
  float* n_mem = p.normaliser + unit * dim;

  auto load4 = [&](int row, float* s) {
    const float* src = S + (size_t)row * vdim + 4 * cq;
    if (vec) {
      const float4 v = *reinterpret_cast<const float4*>(src);
      s[0] = v.x; s[1] = v.y; s[2] = v.z; s[3] = v.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] = 4 * cq + e < vdim ? src[e] : 0.0f;
    }
  };
  auto store4 = [&](int row, const float* s) {
    float* dst = S + (size_t)row * vdim + 4 * cq;
    if (vec) {
      *reinterpret_cast<float4*>(dst) = make_float4(s[0], s[1], s[2], s[3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (4 * cq + e < vdim) dst[e] = s[e];
    }
  };

  float s[R > 0 ? R : 1][4];
  if (R > 0 && active) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int row = rg + i * row_groups;
      if (row < dim) load4(row, s[i]);
    }
  }
  for (int d = tid; d < dim; d += blockDim.x) ns[d] = n_mem[d];
  float m = p.maximum[unit];

  for (int t = first; t < last; ++t) {
    const T* row_t = reinterpret_cast<const T*>(p.rows) + (size_t)t * p.ld;
    const T* q_t = row_t + (size_t)head * dim;
    const T* k_t = row_t + (size_t)(p.heads + head) * dim;
    const T* v_t = row_t + (size_t)2 * p.heads * dim + (size_t)head * vdim;
    for (int d = tid; d < dim; d += blockDim.x) {
      qs[d] = to_float<T>(q_t[d]) * p.q_scale;
      ks[d] = to_float<T>(k_t[d]);
    }
    for (int c = tid; c < 4 * quads; c += blockDim.x) vs[c] = c < vdim ? to_float<T>(v_t[c]) : 0.0f;
    // every thread works the gates out for itself
    const float log_i = soft_cap_m(p.gates[(size_t)t * p.ld_gates + head], p.cap);
    const float log_f = log_sigmoid_m(soft_cap_m(p.gates[(size_t)t * p.ld_gates + p.heads + head], p.cap));
    const float m_new = fmaxf(log_f + m, log_i);
    const float keep = expf(log_f + m - m_new), write = expf(log_i - m_new);
    m = m_new;
    __syncthreads();
    float dot = 0.0f;
    for (int d = tid; d < dim; d += blockDim.x) {
      const float n = fmaf(keep, ns[d], write * ks[d]);
      ns[d] = n;
      dot = fmaf(n, qs[d], dot);
    }
    if (active) {
      const float4 v = *reinterpret_cast<const float4*>(vs + 4 * cq);
      float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      auto update = [&](int row, float* x) {
        const float u = write * ks[row], q = qs[row];
        x[0] = fmaf(keep, x[0], u * v.x);
        x[1] = fmaf(keep, x[1], u * v.y);
        x[2] = fmaf(keep, x[2], u * v.z);
        x[3] = fmaf(keep, x[3], u * v.w);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] = fmaf(x[e], q, acc[e]);
      };
      if (R > 0) {
#pragma unroll
        for (int i = 0; i < R; ++i) {
          const int row = rg + i * row_groups;
          if (row < dim) update(row, s[i]);
        }
      } else {
        for (int row = rg; row < dim; row += row_groups) {
          float x[4];
          load4(row, x);
          update(row, x);
          store4(row, x);
        }
      }
      *reinterpret_cast<float4*>(part + (size_t)rg * 4 * quads + 4 * cq) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    }
    const float den = block_sum(dot, scratch);                 // its barriers also order `part`
    const float inv = 1.0f / (fmaxf(fabsf(den), expf(-m)) + DENOMINATOR_FLOOR);
    float square = 0.0f;
    for (int c = tid; c < vdim; c += blockDim.x) {
      float o = 0.0f;
      for (int g = 0; g < row_groups; ++g) o += part[(size_t)g * 4 * quads + c];
      o *= inv;
      os[c] = o;
      square = fmaf(o, o, square);
    }
    const float factor = 1.0f / sqrtf(block_sum(square, scratch) / (float)vdim + p.eps);
    const T* g_t = row_t + (size_t)2 * p.heads * dim + (size_t)(p.heads + head) * vdim;
    T* dst = reinterpret_cast<T*>(p.out) + (size_t)t * p.ldo + (size_t)head * vdim;
    for (int c = tid; c < vdim; c += blockDim.x)
      dst[c] = from_float<T>(os[c] * factor * p.norm_w[(size_t)head * vdim + c] * sigmoid_m(to_float<T>(g_t[c])));
  }
  if (R > 0 && active) {
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int row = rg + i * row_groups;
      if (row < dim) store4(row, s[i]);
    }
  }
  for (int d = tid; d < dim; d += blockDim.x) n_mem[d] = ns[d];      // each thread its own elements
  if (tid == 0) p.maximum[unit] = m;
}

// ---------------------------------------------------------------------------------------------------------------
// portions in chunks
constexpr int CHUNK = 64;
constexpr int CHUNK_THREADS = 128;
constexpr int CHUNK_MAX_VALUES = 128, CHUNK_MAX_KEYS = 256;

struct ChunkParams {
  MlstmParams m;
  double* g;                   // [heads, tokens]: log input gate less the running sum of log forget gates
  double* top;                 // [heads, tokens]: M
  float* floor;                // [heads, tokens]: exp(-m)
  double* start;               // [num_seqs, heads]: the maximum a portion starts with
  float* own;                  // [wave, heads, dim, vdim]: a chunk's own contribution
  __nv_bfloat16* before;       // [3][wave, heads, dim, vdim]: the state before a chunk, in three parts
  float* norm_own;             // [wave, heads, dim]: a chunk's own contribution to the normaliser; the carry puts the
                               // normaliser before the chunk in its place
  int tokens, num_seqs;
  int first_chunk, wave;       // the chunks this launch is about, out of all portions' chunks in order
};

__device__ __forceinline__ int chunks_of(const MlstmParams& m, int seq) {
  const int n = m.q_start[seq + 1] - m.q_start[seq];
  return n > m.longest ? (n + CHUNK - 1) / CHUNK : 0;
}

// Which portion a chunk belongs to, its first token, how many it has and which of its portion's chunks it is.
struct ChunkPlace {
  int seq, first, count, index;
};
__device__ __forceinline__ ChunkPlace place_of(const ChunkParams& p, int chunk) {
  ChunkPlace out{-1, 0, 0, 0};
  for (int s = 0; s < p.num_seqs; ++s) {
    const int n = chunks_of(p.m, s);
    if (chunk < n) {
      out.seq = s;
      out.index = chunk;
      out.first = p.m.q_start[s] + chunk * CHUNK;
      out.count = min(CHUNK, p.m.q_start[s + 1] - out.first);
      return out;
    }
    chunk -= n;
  }
  return out;
}
// M right before a chunk.
__device__ __forceinline__ double top_before(const ChunkParams& p, int seq, int head, int first, int index) {
  return index == 0 ? p.start[(size_t)seq * p.m.heads + head] : p.top[(size_t)head * p.tokens + first - 1];
}

// A float32 number as the sum of three bfloat16 ones.
__device__ __forceinline__ void three_parts(float x, float& a, float& b, float& c) {
  a = __bfloat162float(__float2bfloat16_rn(x));
  b = __bfloat162float(__float2bfloat16_rn(x - a));
  c = x - a - b;
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ uint32_t shared_address(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldm4(uint32_t at, uint32_t& a, uint32_t& b, uint32_t& c, uint32_t& d) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(a), "=r"(b), "=r"(c), "=r"(d) : "r"(at));
}
__device__ __forceinline__ void ldm4_t(uint32_t at, uint32_t& a, uint32_t& b, uint32_t& c, uint32_t& d) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(a), "=r"(b), "=r"(c), "=r"(d) : "r"(at));
}
__device__ __forceinline__ void mma16(float c[4], const uint32_t a[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void copy16(void* dst, const void* src, bool real) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(shared_address(dst)), "l"(src), "r"(real ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copies_sent() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copies_landed() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

// rows [count of 64][width] of a chunk into shared memory [64][pitch], zeros beyond the chunk and beyond the width
__device__ __forceinline__ void copy_rows(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, long long ld, int count, int width,
                                          int padded) {
  const int units = padded / 8;
  for (int r = threadIdx.x >> 4; r < CHUNK; r += CHUNK_THREADS / 16)          // sixteen lanes to a row
    for (int u = threadIdx.x & 15; u < units; u += 16) {
      const bool real = r < count && u * 8 < width;
      copy16(dst + r * pitch + u * 8, real ? src + (size_t)r * ld + u * 8 : src, real);
    }
}

constexpr int SCAN_THREADS = 256;

// One block per (head, portion): F, g, M and exp(-m) of its tokens, and its new maximum.
__global__ void __launch_bounds__(SCAN_THREADS) mlstm_gate_scan_kernel(const ChunkParams p) {
  __shared__ double totals[SCAN_THREADS / 32];
  pdl_trigger();
  const int head = blockIdx.x, seq = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int first = p.m.q_start[seq], last = p.m.q_start[seq + 1];
  const size_t unit = (size_t)p.m.slots[seq] * p.m.heads + head;
  pdl_wait();
  if (chunks_of(p.m, seq) == 0) return;
  const double start = p.m.maximum[unit];
  double sum_before = 0.0, top_so_far = start;
  for (int base = first; base < last; base += SCAN_THREADS) {
    const int t = base + threadIdx.x;
    const bool live = t < last;
    float log_i = -INFINITY, log_f = 0.0f;
    if (live) {
      const float* z = p.m.gates + (size_t)t * p.m.ld_gates;
      log_i = soft_cap_m(z[head], p.m.cap);
      log_f = log_sigmoid_m(soft_cap_m(z[p.m.heads + head], p.m.cap));
    }
    double sum = log_f;
#pragma unroll
    for (int step = 1; step < 32; step <<= 1) {
      const double other = __shfl_up_sync(0xffffffffu, sum, step);
      if (lane >= step) sum += other;
    }
    if (lane == 31) totals[warp] = sum;
    __syncthreads();
    double all = sum_before;
    for (int w = 0; w < SCAN_THREADS / 32; ++w) {
      if (w < warp) sum += totals[w];
      all += totals[w];
    }
    sum += sum_before;
    __syncthreads();
    const double g = (double)log_i - sum;
    double top = g;
#pragma unroll
    for (int step = 1; step < 32; step <<= 1) {
      const double other = __shfl_up_sync(0xffffffffu, top, step);
      if (lane >= step) top = fmax(top, other);
    }
    if (lane == 31) totals[warp] = top;
    __syncthreads();
    double most = top_so_far;
    for (int w = 0; w < SCAN_THREADS / 32; ++w) {
      if (w < warp) top = fmax(top, totals[w]);
      most = fmax(most, totals[w]);
    }
    top = fmax(top, top_so_far);
    __syncthreads();
    if (live) {
      const size_t at = (size_t)head * p.tokens + t;
      p.g[at] = g;
      p.top[at] = top;
      p.floor[at] = expf((float)-(top + sum));
      if (t == last - 1) p.m.maximum[unit] = (float)(top + sum);
    }
    sum_before = all;
    top_so_far = most;
  }
  if (threadIdx.x == 0) p.start[(size_t)seq * p.m.heads + head] = start;
}

// A chunk's own contribution to its head's state and normaliser, as seen at its last token.  VD: values, padded.
template <int VD>
__global__ void __launch_bounds__(CHUNK_THREADS) mlstm_chunk_write_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char chunk_smem[];
  pdl_trigger();
  const int head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dim = p.m.dim, vdim = p.m.vdim;
  const int kd = (dim + 15) / 16 * 16, k_pitch = kd + 8;
  constexpr int V_PITCH = VD + 8;
  __nv_bfloat16* vs = reinterpret_cast<__nv_bfloat16*>(chunk_smem);     // [64][V_PITCH]
  __nv_bfloat16* kw = vs + CHUNK * V_PITCH;                             // [3][64][k_pitch]: factor times key
  float* factor = reinterpret_cast<float*>(kw + 3 * CHUNK * k_pitch);   // [64]
  const ChunkPlace at = place_of(p, p.first_chunk + blockIdx.x);
  pdl_wait();
  if (at.seq < 0) return;
  const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(p.m.rows) + (size_t)at.first * p.m.ld;
  const __nv_bfloat16* k_rows = rows + (size_t)(p.m.heads + head) * dim;
  copy_rows(vs, V_PITCH, rows + (size_t)2 * p.m.heads * dim + (size_t)head * vdim, p.m.ld, at.count, vdim, VD);
  copies_sent();
  const size_t line = (size_t)head * p.tokens + at.first;
  if (tid < CHUNK) factor[tid] = tid < at.count ? expf((float)(p.g[line + tid] - p.top[line + at.count - 1])) : 0.0f;
  __syncthreads();
  for (int e = tid; e < CHUNK * (kd / 8); e += CHUNK_THREADS) {
    const int r = e / (kd / 8), u = e - r * (kd / 8);
    uint4 raw = make_uint4(0u, 0u, 0u, 0u);
    if (r < at.count && u * 8 < dim) raw = *reinterpret_cast<const uint4*>(k_rows + (size_t)r * p.m.ld + u * 8);
    const __nv_bfloat162* two = reinterpret_cast<const __nv_bfloat162*>(&raw);
    const float w = factor[r];
    uint32_t parts[3][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(two[i]);
      float a0, b0, c0, a1, b1, c1;
      three_parts(f.x * w, a0, b0, c0);
      three_parts(f.y * w, a1, b1, c1);
      parts[0][i] = pack2(a0, a1);
      parts[1][i] = pack2(b0, b1);
      parts[2][i] = pack2(c0, c1);
    }
#pragma unroll
    for (int part = 0; part < 3; ++part)
      *reinterpret_cast<uint4*>(kw + ((size_t)part * CHUNK + r) * k_pitch + u * 8) =
          make_uint4(parts[part][0], parts[part][1], parts[part][2], parts[part][3]);
  }
  copies_landed<0>();
  __syncthreads();
  const size_t unit = (size_t)blockIdx.x * p.m.heads + head;
  for (int d = tid; d < dim; d += CHUNK_THREADS) {
    float sum = 0.0f;
    for (int r = 0; r < at.count; ++r) {
      const __nv_bfloat16* src = kw + (size_t)r * k_pitch + d;
      sum += __bfloat162float(src[0]) + (__bfloat162float(src[(size_t)CHUNK * k_pitch]) + __bfloat162float(src[(size_t)2 * CHUNK * k_pitch]));
    }
    p.norm_own[unit * dim + d] = sum;
  }
  float* own = p.own + unit * dim * vdim;
  const int g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3;
  for (int tile = warp; tile < kd / 16; tile += CHUNK_THREADS / 32) {
    float acc[VD / 8][4];
#pragma unroll
    for (int n = 0; n < VD / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[n][e] = 0.0f;
#pragma unroll
    for (int ks = 0; ks < CHUNK / 16; ++ks) {
      uint32_t a[3][4];
#pragma unroll
      for (int part = 0; part < 3; ++part)
        ldm4_t(shared_address(kw + ((size_t)part * CHUNK + ks * 16 + (mi >> 1) * 8 + (lane & 7)) * k_pitch + tile * 16 + (mi & 1) * 8),
               a[part][0], a[part][1], a[part][2], a[part][3]);
#pragma unroll
      for (int n = 0; n < VD / 8; n += 2) {
        uint32_t b0, b1, b2, b3;
        ldm4_t(shared_address(vs + (ks * 16 + (mi & 1) * 8 + (lane & 7)) * V_PITCH + (n + (mi >> 1)) * 8), b0, b1, b2, b3);
#pragma unroll
        for (int part = 2; part >= 0; --part) {
          mma16(acc[n], a[part], b0, b1);
          mma16(acc[n + 1], a[part], b2, b3);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = tile * 16 + g8 + 8 * i;
      if (row >= dim) continue;
#pragma unroll
      for (int n = 0; n < VD / 8; ++n)
        if (n * 8 + 2 * t4 < vdim)
          *reinterpret_cast<float2*>(own + (size_t)row * vdim + n * 8 + 2 * t4) = make_float2(acc[n][2 * i], acc[n][2 * i + 1]);
    }
  }
}

// The state from chunk to chunk: S <- exp(M_before - M_end) S + the chunk's own; what it was before every chunk is left in
// three bfloat16 parts for the readout.  Four entries of a head's state per thread, then the normaliser.
__global__ void __launch_bounds__(256) mlstm_chunk_carry_kernel(const ChunkParams p) {
  pdl_trigger();
  const int head = blockIdx.y, seq = blockIdx.z;
  const int dim = p.m.dim, vdim = p.m.vdim;
  int base = 0;
  for (int s = 0; s < seq; ++s) base += chunks_of(p.m, s);
  const int mine = chunks_of(p.m, seq);
  const int from = max(base, p.first_chunk), to = min(base + mine, p.first_chunk + p.wave);
  const size_t entries = (size_t)dim * vdim;
  const size_t quads = entries / 4;
  const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const int first = p.m.q_start[seq], last = p.m.q_start[seq + 1];
  const size_t slot_unit = (size_t)p.m.slots[seq] * p.m.heads + head;
  const size_t plane = (size_t)p.wave * p.m.heads * entries;
  pdl_wait();
  if (from >= to || e >= quads + dim) return;
  const double* top = p.top + (size_t)head * p.tokens;
  double before = top_before(p, seq, head, first + (from - base) * CHUNK, from - base);
  if (e < quads) {
    float4* state = reinterpret_cast<float4*>(p.m.state + slot_unit * entries) + e;
    float4 s = *state;
    float4 next = reinterpret_cast<const float4*>(p.own + ((size_t)(from - p.first_chunk) * p.m.heads + head) * entries)[e];
    for (int c = from; c < to; ++c) {
      const float4 own = next;
      if (c + 1 < to) next = reinterpret_cast<const float4*>(p.own + ((size_t)(c + 1 - p.first_chunk) * p.m.heads + head) * entries)[e];
      const double end = top[min(first + (c - base + 1) * CHUNK, last) - 1];
      const float keep = expf((float)(before - end));
      before = end;
      float a[4], b[4], d[4];
      three_parts(s.x, a[0], b[0], d[0]);
      three_parts(s.y, a[1], b[1], d[1]);
      three_parts(s.z, a[2], b[2], d[2]);
      three_parts(s.w, a[3], b[3], d[3]);
      const size_t out = ((size_t)(c - p.first_chunk) * p.m.heads + head) * entries + 4 * e;
      *reinterpret_cast<uint2*>(p.before + out) = make_uint2(pack2(a[0], a[1]), pack2(a[2], a[3]));
      *reinterpret_cast<uint2*>(p.before + plane + out) = make_uint2(pack2(b[0], b[1]), pack2(b[2], b[3]));
      *reinterpret_cast<uint2*>(p.before + 2 * plane + out) = make_uint2(pack2(d[0], d[1]), pack2(d[2], d[3]));
      s.x = fmaf(keep, s.x, own.x);
      s.y = fmaf(keep, s.y, own.y);
      s.z = fmaf(keep, s.z, own.z);
      s.w = fmaf(keep, s.w, own.w);
    }
    *state = s;
  } else {
    const int d = (int)(e - quads);
    float* normaliser = p.m.normaliser + slot_unit * dim + d;
    float n = *normaliser;
    for (int c = from; c < to; ++c) {
      float* at = p.norm_own + ((size_t)(c - p.first_chunk) * p.m.heads + head) * dim + d;
      const float own = *at;
      const double end = top[min(first + (c - base + 1) * CHUNK, last) - 1];
      const float keep = expf((float)(before - end));
      before = end;
      *at = n;
      n = fmaf(keep, n, own);
    }
    *normaliser = n;
  }
}

constexpr int STATE_ROWS = 32;          // rows of the state before a chunk that lie in shared memory at a time (three parts)
// The ring of state rows, and after it in the same place the chunk's keys and values.
__host__ __device__ constexpr int read_ring_elements(int k_pitch, int v_pitch) {
  return 6 * STATE_ROWS * v_pitch > CHUNK * (k_pitch + v_pitch) ? 6 * STATE_ROWS * v_pitch : CHUNK * (k_pitch + v_pitch);
}

// The readout of a chunk: what its own earlier tokens and the state before it give, over the denominator, normalised per
// head, weighted and gated.  Four warps, 16 tokens each.
template <int VD>
__global__ void __launch_bounds__(CHUNK_THREADS) mlstm_chunk_read_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) unsigned char chunk_smem[];
  pdl_trigger();
  const int head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dim = p.m.dim, vdim = p.m.vdim;
  const int kd = (dim + 15) / 16 * 16, k_pitch = kd + 8;
  constexpr int V_PITCH = VD + 8;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(chunk_smem);     // [64][k_pitch]
  __nv_bfloat16* ss = qs + CHUNK * k_pitch;                             // [2][3][STATE_ROWS][V_PITCH]; once the state is read:
  __nv_bfloat16* ks = ss;                                               // [64][k_pitch]
  __nv_bfloat16* vs = ks + CHUNK * k_pitch;                             // [64][V_PITCH]
  double* g_s = reinterpret_cast<double*>(ss + read_ring_elements(k_pitch, V_PITCH));    // [64]
  float* n_s = reinterpret_cast<float*>(g_s + CHUNK);                   // [kd]
  float* den_s = n_s + kd;                                              // [64]
  const ChunkPlace at = place_of(p, p.first_chunk + blockIdx.x);
  const size_t line = (size_t)head * p.tokens + at.first;
  const size_t entries = (size_t)dim * vdim;
  const size_t unit = (size_t)blockIdx.x * p.m.heads + head;
  const size_t plane = (size_t)p.wave * p.m.heads * entries;
  pdl_wait();
  if (at.seq < 0) return;
  const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(p.m.rows) + (size_t)at.first * p.m.ld;
  copy_rows(qs, k_pitch, rows + (size_t)head * dim, p.m.ld, at.count, dim, kd);
  auto fetch_state = [&](int slice) {
    constexpr int UNITS = VD / 8;
    __nv_bfloat16* dst = ss + (slice & 1) * 3 * STATE_ROWS * V_PITCH;
    const __nv_bfloat16* src = p.before + unit * entries;
#pragma unroll
    for (int part = 0; part < 3; ++part, src += plane)
#pragma unroll
      for (int r = tid >> 4; r < STATE_ROWS; r += CHUNK_THREADS / 16) {
        const int row = slice * STATE_ROWS + r, u = tid & 15;
        if (u >= UNITS) continue;
        const bool real = row < dim && u * 8 < vdim;
        copy16(dst + (part * STATE_ROWS + r) * V_PITCH + u * 8, real ? src + (size_t)row * vdim + u * 8 : src, real);
      }
    copies_sent();
  };
  const int slices = (kd + STATE_ROWS - 1) / STATE_ROWS;
  fetch_state(0);                                          // one group with q
  if (tid < CHUNK) g_s[tid] = tid < at.count ? p.g[line + tid] : 0.0;
  for (int d = tid; d < kd; d += CHUNK_THREADS) n_s[d] = d < dim ? p.norm_own[unit * dim + d] : 0.0f;
  const double before = top_before(p, at.seq, head, at.first, at.index);
  const int g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3;
  double top[2];
  float inter[2];
  int row[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    row[i] = warp * 16 + g8 + 8 * i;
    top[i] = row[i] < at.count ? p.top[line + row[i]] : 0.0;
    inter[i] = row[i] < at.count ? expf((float)(before - top[i])) * p.m.q_scale : 0.0f;
  }

  float acc[VD / 8][4];
#pragma unroll
  for (int n = 0; n < VD / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.0f;
  // what the state before the chunk gives
  for (int slice = 0; slice < slices; ++slice) {
    if (slice + 1 < slices) {
      fetch_state(slice + 1);
      copies_landed<1>();
    } else {
      copies_landed<0>();
    }
    __syncthreads();
    if (slice == 0) {
      // the normaliser before the chunk: two threads to a token
      const int r = tid >> 1, half = tid & 1;
      float dot = 0.0f;
      for (int d = half * (kd / 2); d < (half + 1) * (kd / 2); ++d) dot = fmaf(__bfloat162float(qs[r * k_pitch + d]), n_s[d], dot);
      dot += __shfl_xor_sync(0xffffffffu, dot, 1);
      if (half == 0) den_s[r] = dot;
    }
    const __nv_bfloat16* part_s = ss + (slice & 1) * 3 * STATE_ROWS * V_PITCH;
#pragma unroll
    for (int step = 0; step < STATE_ROWS / 16; ++step) {
      const int d0 = slice * STATE_ROWS + step * 16;
      if (d0 >= kd) break;
      uint32_t a[4];
      ldm4(shared_address(qs + (warp * 16 + (mi & 1) * 8 + (lane & 7)) * k_pitch + d0 + (mi >> 1) * 8), a[0], a[1], a[2], a[3]);
#pragma unroll
      for (int n = 0; n < VD / 8; n += 2) {
#pragma unroll
        for (int part = 2; part >= 0; --part) {
          uint32_t b0, b1, b2, b3;
          ldm4_t(shared_address(part_s + (part * STATE_ROWS + step * 16 + (mi & 1) * 8 + (lane & 7)) * V_PITCH + (n + (mi >> 1)) * 8), b0,
                 b1, b2, b3);
          mma16(acc[n], a, b0, b1);
          mma16(acc[n + 1], a, b2, b3);
        }
      }
    }
    __syncthreads();                                       // the buffer is copied into again two slices on
  }
  copy_rows(ks, k_pitch, rows + (size_t)(p.m.heads + head) * dim, p.m.ld, at.count, dim, kd);
  copies_sent();
  copy_rows(vs, V_PITCH, rows + (size_t)2 * p.m.heads * dim + (size_t)head * vdim, p.m.ld, at.count, vdim, VD);
  copies_sent();
#pragma unroll
  for (int n = 0; n < VD / 8; ++n) {
    acc[n][0] *= inter[0]; acc[n][1] *= inter[0];
    acc[n][2] *= inter[1]; acc[n][3] *= inter[1];
  }
  // what the chunk's own tokens give: q k^T, the factors, times v; a warp needs the first 16 (warp + 1) of them
  float sc[CHUNK / 8][4];
#pragma unroll
  for (int n = 0; n < CHUNK / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) sc[n][e] = 0.0f;
  copies_landed<1>();
  __syncthreads();
  for (int d0 = 0; d0 < kd; d0 += 16) {
    uint32_t a[4];
    ldm4(shared_address(qs + (warp * 16 + (mi & 1) * 8 + (lane & 7)) * k_pitch + d0 + (mi >> 1) * 8), a[0], a[1], a[2], a[3]);
#pragma unroll
    for (int n = 0; n < CHUNK / 8; n += 2) {
      if (n > 2 * warp) continue;
      uint32_t b0, b1, b2, b3;
      ldm4(shared_address(ks + ((n + (mi >> 1)) * 8 + (lane & 7)) * k_pitch + d0 + (mi & 1) * 8), b0, b1, b2, b3);
      mma16(sc[n], a, b0, b1);
      mma16(sc[n + 1], a, b2, b3);
    }
  }
  float den[2] = {0.0f, 0.0f};
#pragma unroll
  for (int n = 0; n < CHUNK / 8; ++n) {
    if (n > 2 * warp + 1) continue;
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int s = n * 8 + 2 * t4 + e;
        float w = 0.0f;
        if (s <= row[i] && row[i] < at.count) w = sc[n][2 * i + e] * p.m.q_scale * expf((float)(g_s[s] - top[i]));
        sc[n][2 * i + e] = w;
        den[i] += w;
      }
  }
  copies_landed<0>();
  __syncthreads();
#pragma unroll
  for (int ksub = 0; ksub < CHUNK / 16; ++ksub) {
    if (ksub > warp) continue;
    uint32_t a[3][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      // fragment register j: rows g8 (+ 8 for odd j), columns 2 t4 (+ 8 for j > 1)
      const float x = sc[2 * ksub + (j >> 1)][2 * (j & 1)], y = sc[2 * ksub + (j >> 1)][2 * (j & 1) + 1];
      float x0, x1, x2, y0, y1, y2;
      three_parts(x, x0, x1, x2);
      three_parts(y, y0, y1, y2);
      a[0][j] = pack2(x0, y0);
      a[1][j] = pack2(x1, y1);
      a[2][j] = pack2(x2, y2);
    }
#pragma unroll
    for (int n = 0; n < VD / 8; n += 2) {
      uint32_t b0, b1, b2, b3;
      ldm4_t(shared_address(vs + (ksub * 16 + (mi & 1) * 8 + (lane & 7)) * V_PITCH + (n + (mi >> 1)) * 8), b0, b1, b2, b3);
#pragma unroll
      for (int part = 2; part >= 0; --part) {
        mma16(acc[n], a[part], b0, b1);
        mma16(acc[n + 1], a[part], b2, b3);
      }
    }
  }
  const __nv_bfloat16* gate_rows = rows + (size_t)2 * p.m.heads * dim + (size_t)(p.m.heads + head) * vdim;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.m.out) + (size_t)at.first * p.m.ldo + (size_t)head * vdim;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    den[i] += __shfl_xor_sync(0xffffffffu, den[i], 1);
    den[i] += __shfl_xor_sync(0xffffffffu, den[i], 2);
    const bool live = row[i] < at.count;
    const float total = live ? den[i] + inter[i] * den_s[row[i]] : 0.0f;
    const float inv = live ? 1.0f / (fmaxf(fabsf(total), p.floor[line + row[i]]) + DENOMINATOR_FLOOR) : 0.0f;
    float square = 0.0f;
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) {
      acc[n][2 * i] *= inv;
      acc[n][2 * i + 1] *= inv;
      square = fmaf(acc[n][2 * i], acc[n][2 * i], fmaf(acc[n][2 * i + 1], acc[n][2 * i + 1], square));
    }
    square += __shfl_xor_sync(0xffffffffu, square, 1);
    square += __shfl_xor_sync(0xffffffffu, square, 2);
    if (!live) continue;
    const float factor = 1.0f / sqrtf(square / (float)vdim + p.m.eps);
#pragma unroll
    for (int n = 0; n < VD / 8; ++n) {
      const int c = n * 8 + 2 * t4;
      if (c >= vdim) continue;
      const float2 gate = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate_rows + (size_t)row[i] * p.m.ld + c));
      const float2 w = *reinterpret_cast<const float2*>(p.m.norm_w + (size_t)head * vdim + c);
      *reinterpret_cast<uint32_t*>(out + (size_t)row[i] * p.m.ldo + c) =
          pack2(acc[n][2 * i] * factor * w.x * sigmoid_fast(gate.x), acc[n][2 * i + 1] * factor * w.y * sigmoid_fast(gate.y));
    }
  }
}

bool chunk_shapes(int dim, int vdim) {
  return dim % 8 == 0 && vdim % 8 == 0 && dim <= CHUNK_MAX_KEYS && vdim <= CHUNK_MAX_VALUES;
}

template <int VD>
int launch_chunks(ChunkParams p, int chunks, cudaStream_t stream) {
  const int kd = (p.m.dim + 15) / 16 * 16;
  const size_t write_smem = ((size_t)CHUNK * (VD + 8) + (size_t)3 * CHUNK * (kd + 8)) * 2 + CHUNK * sizeof(float);
  const size_t read_smem = ((size_t)CHUNK * (kd + 8) + (size_t)read_ring_elements(kd + 8, VD + 8)) * 2 +
                           CHUNK * sizeof(double) + (size_t)(kd + CHUNK) * sizeof(float);
  static size_t configured = 0;
  if (write_smem > configured || read_smem > configured) {
    const size_t most = write_smem > read_smem ? write_smem : read_smem;
    cudaError_t err = cudaFuncSetAttribute(mlstm_chunk_write_kernel<VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most);
    if (err == cudaSuccess) err = cudaFuncSetAttribute(mlstm_chunk_read_kernel<VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most);
    if (err != cudaSuccess) {
      tge_set_error("mlstm_chunks: cannot reserve %zu bytes of shared memory: %s", most, cudaGetErrorString(err));
      return -2;
    }
    configured = most;
  }
  tge_launch(mlstm_gate_scan_kernel, dim3(p.m.heads, p.num_seqs), dim3(SCAN_THREADS), 0, stream, p);
  int kernels = 1;
  const size_t work = (size_t)p.m.dim * p.m.vdim / 4 + p.m.dim;
  const int wave = p.wave;
  for (int first = 0; first < chunks; first += wave) {
    p.first_chunk = first;
    const int count = chunks - first < wave ? chunks - first : wave;
    tge_launch(mlstm_chunk_write_kernel<VD>, dim3(count, p.m.heads), dim3(CHUNK_THREADS), write_smem, stream, p);
    tge_launch(mlstm_chunk_carry_kernel, dim3((unsigned)((work + 255) / 256), p.m.heads, p.num_seqs), dim3(256), 0, stream, p);
    tge_launch(mlstm_chunk_read_kernel<VD>, dim3(count, p.m.heads), dim3(CHUNK_THREADS), read_smem, stream, p);
    kernels += 3;
  }
  return tge_launched("mlstm_chunks", kernels);
}

template <typename T>
int launch_step(const MlstmParams& p, int num_seqs, cudaStream_t stream) {
  const int quads = (p.vdim + 3) / 4;
  int threads = 256;
  auto rows_at = [&](int n) { return n < quads ? 1 << 30 : (p.dim + n / quads - 1) / (n / quads); };
  while (threads < 1024 && rows_at(threads) > 16) threads *= 2;
  TGE_REQUIRE(quads <= threads, "mlstm_step: values of %d numbers (up to %d)", p.vdim, 4 * threads);
  const int rows = rows_at(threads);
  const size_t smem = ((size_t)3 * ((p.dim + 3) & ~3) + 8 * quads + (size_t)(threads / quads) * 4 * quads) * sizeof(float);
  TGE_REQUIRE(smem <= 48 * 1024, "mlstm_step: heads of %d x %d need %zu bytes of shared memory", p.dim, p.vdim, smem);
  const dim3 grid(p.heads, num_seqs), block(threads);
  if (rows <= 2) tge_launch(mlstm_step_kernel<T, 2>, grid, block, smem, stream, p);
  else if (rows <= 4) tge_launch(mlstm_step_kernel<T, 4>, grid, block, smem, stream, p);
  else if (rows <= 8 && threads <= 512) tge_launch(mlstm_step_kernel<T, 8>, grid, block, smem, stream, p);
  else if (rows <= 16 && threads <= 512) tge_launch(mlstm_step_kernel<T, 16>, grid, block, smem, stream, p);
  else tge_launch(mlstm_step_kernel<T, 0>, grid, block, smem, stream, p);
  return tge_launched("mlstm_step", 1);
}

}  // namespace

// rows: run dtype [tokens, ld] = [q | k | v | g]; gates float32 [tokens, ld_gates] = [zi | zf]; the states' rows
// slots[s] are read and written; out: run dtype [tokens, ldo].  Portions longer than `longest` tokens are not touched.
TGE_API int tge_mlstm_step(const void* rows, int is_bf16, long long ld, const float* gates, long long ld_gates,
                           const float* norm_w, float* state, float* normaliser, float* maximum, const int* slots,
                           const int* q_start, void* out, long long ldo, int num_seqs, int heads, int dim, int vdim,
                           int longest, float cap, float q_scale, float eps, cudaStream_t stream) {
  TGE_REQUIRE(num_seqs >= 0 && num_seqs <= 65535 && heads > 0 && dim > 0 && vdim > 0, "mlstm_step: bad sizes");
  TGE_REQUIRE(ld >= 2LL * heads * (dim + vdim) && ld_gates >= 2LL * heads && ldo >= (long long)heads * vdim,
              "mlstm_step: rows of %lld and %lld numbers into rows of %lld", ld, ld_gates, ldo);
  TGE_REQUIRE(cap > 0.0f && eps > 0.0f, "mlstm_step: the cap and eps must be positive");
  TGE_REQUIRE(((uintptr_t)state & 15) == 0, "mlstm_step: the state must start on 16 bytes");
  if (num_seqs == 0) return 0;
  MlstmParams p;
  p.rows = rows; p.ld = ld; p.gates = gates; p.ld_gates = ld_gates; p.norm_w = norm_w; p.state = state;
  p.normaliser = normaliser; p.maximum = maximum; p.slots = slots; p.q_start = q_start; p.out = out; p.ldo = ldo;
  p.heads = heads; p.dim = dim; p.vdim = vdim; p.longest = longest; p.cap = cap; p.q_scale = q_scale; p.eps = eps;
  return is_bf16 ? launch_step<__nv_bfloat16>(p, num_seqs, stream) : launch_step<float>(p, num_seqs, stream);
}

// Whether portions of many tokens may go through the chunk kernels at these sizes.
TGE_API int tge_mlstm_chunks_supported(int dim, int vdim) { return chunk_shapes(dim, vdim) ? 1 : 0; }

// Portions of more than `longest` tokens, bfloat16, in chunks of 64 (see the head of this file); shorter ones are not
// touched.  Scratch: g and top float64 [heads, tokens], floor float32 [heads, tokens], start float64 [num_seqs, heads],
// own float32 [wave, heads, dim, vdim], before bfloat16 [3, wave, heads, dim, vdim], norm_own float32 [wave, heads, dim];
// `chunks` is at least the number of chunks all portions have, `wave` how many are worked on at a time.
TGE_API int tge_mlstm_chunks(const void* rows, long long ld, const float* gates, long long ld_gates, const float* norm_w,
                             float* state, float* normaliser, float* maximum, const int* slots, const int* q_start, void* out,
                             long long ldo, int num_seqs, int tokens, int heads, int dim, int vdim, int longest, float cap,
                             float q_scale, float eps, double* g, double* top, float* floor, double* start, float* own,
                             void* before, float* norm_own, int chunks, int wave, cudaStream_t stream) {
  TGE_REQUIRE(num_seqs >= 0 && num_seqs <= 65535 && heads > 0 && heads <= 65535 && tokens >= 0 && chunks >= 0 && wave > 0,
              "mlstm_chunks: bad sizes");
  TGE_REQUIRE(chunk_shapes(dim, vdim), "mlstm_chunks: heads of %d x %d (multiples of 8 up to %d x %d)", dim, vdim, CHUNK_MAX_KEYS,
              CHUNK_MAX_VALUES);
  TGE_REQUIRE(ld >= 2LL * heads * (dim + vdim) && ld % 8 == 0 && ld_gates >= 2LL * heads && ldo >= (long long)heads * vdim && ldo % 2 == 0,
              "mlstm_chunks: rows of %lld and %lld numbers into rows of %lld", ld, ld_gates, ldo);
  TGE_REQUIRE(cap > 0.0f && eps > 0.0f && longest >= 0, "mlstm_chunks: the cap and eps must be positive");
  TGE_REQUIRE((((uintptr_t)rows | (uintptr_t)state | (uintptr_t)own | (uintptr_t)before) & 15) == 0 && ((uintptr_t)norm_w & 7) == 0 &&
                  ((uintptr_t)out & 3) == 0, "mlstm_chunks: misaligned tensors");
  if (num_seqs == 0 || tokens == 0 || chunks == 0) return 0;
  ChunkParams p;
  p.m.rows = rows; p.m.ld = ld; p.m.gates = gates; p.m.ld_gates = ld_gates; p.m.norm_w = norm_w; p.m.state = state;
  p.m.normaliser = normaliser; p.m.maximum = maximum; p.m.slots = slots; p.m.q_start = q_start; p.m.out = out; p.m.ldo = ldo;
  p.m.heads = heads; p.m.dim = dim; p.m.vdim = vdim; p.m.longest = longest; p.m.cap = cap; p.m.q_scale = q_scale; p.m.eps = eps;
  p.g = g; p.top = top; p.floor = floor; p.start = start; p.own = own; p.before = (__nv_bfloat16*)before; p.norm_own = norm_own;
  p.tokens = tokens; p.num_seqs = num_seqs; p.first_chunk = 0; p.wave = wave;
  if (vdim <= 32) return launch_chunks<32>(p, chunks, stream);
  if (vdim <= 64) return launch_chunks<64>(p, chunks, stream);
  if (vdim <= 96) return launch_chunks<96>(p, chunks, stream);
  return launch_chunks<128>(p, chunks, stream);
}
