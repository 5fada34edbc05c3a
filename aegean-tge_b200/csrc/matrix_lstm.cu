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
//                 costs one read and one write of its state and nothing else.
//
// Gates, the maximum, the normaliser, the state and the readout are float32 in both number formats; q, k, v and g come
// from a product in the run's format.
#include "common.cuh"

namespace {

constexpr float DENOMINATOR_FLOOR = 1e-6f;

__device__ __forceinline__ float sigmoid_m(float z) { return 1.0f / (1.0f + expf(-z)); }
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
  if (first >= last || last - first > p.longest) return;
  const int dim = p.dim, vdim = p.vdim;
  const int quads = (vdim + 3) / 4, row_groups = blockDim.x / quads;
  const int cq = tid % quads, rg = tid / quads;
  const bool active = rg < row_groups;
  const bool vec = (vdim & 3) == 0;
  float* qs = step_smem;                       // [dim]
  float* ks = qs + dim;                        // [dim]
  float* ns = ks + dim;                        // [dim]
  float* vs = ns + dim;                        // [4 quads]
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

  pdl_wait();
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

template <typename T>
int launch_step(const MlstmParams& p, int num_seqs, cudaStream_t stream) {
  const int quads = (p.vdim + 3) / 4;
  int threads = 256;
  auto rows_at = [&](int n) { return n < quads ? 1 << 30 : (p.dim + n / quads - 1) / (n / quads); };
  while (threads < 1024 && rows_at(threads) > 16) threads *= 2;
  TGE_REQUIRE(quads <= threads, "mlstm_step: values of %d numbers (up to %d)", p.vdim, 4 * threads);
  const int rows = rows_at(threads);
  const size_t smem = ((size_t)3 * p.dim + 8 * quads + (size_t)(threads / quads) * 4 * quads) * sizeof(float);
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
