// Kernels of a routed feed-forward (a mixture of small experts) and of activations that stand alone.
//
//  * router_topk      - from float32 router logits: softmax over all outputs or each output's logistic function, the
//                       choice by score + correction inside the best groups of neighbouring outputs (a group's value its
//                       largest such number, or the sum of its two largest), the chosen outputs' plain scores, over their
//                       sum or as they are, times a constant.
//  * activation       - relu(z)^2, or the two-parameter form z > 0: softplus(p) z^2 + z/2, else
//                       (1/2 + softplus(q)) (exp(z) - 1 - z) + z/2, in place on rows of the run dtype.
//  * expert_up / expert_down_add - few tokens (a decode step): every (token, chosen expert) pair reads its expert's
//                       rows directly, one warp per output, and the weighted outputs are added into the float32 stream
//                       in the order of the choice; outputs beyond the experts are identity experts (the input itself).
//  * expert_dense_weigh - a step of some tokens that between them choose most experts anyway: every token goes through
//                       every expert's up matrix in ONE product, this kernel weighs the chosen experts' activated rows
//                       and zeroes the others, and ONE product with all down matrices side by side adds the sum.
//  * expert_sort / expert_gather / expert_combine_add - many tokens: the pairs are grouped by expert so that each
//                       expert's rows form one block of a buffer, which ordinary products then multiply; the last
//                       kernel adds the weighted rows back into the stream, again in the order of the choice.
//
// An expert is relu(up h)^2 or a clamped gated one, min(g, L) sigmoid(alpha min(g, L)) (clamp(u, -L, L) + offset) with
// the gate and up rows interleaved in its first matrix; a choice's weight multiplies the expert's output or its input.
//
// The router, the weights, every accumulation and the sum into the stream are float32.
#include <limits.h>

#include "common.cuh"

namespace {

__device__ __forceinline__ float softplus_f(float z) { return log1pf(expf(-fabsf(z))) + fmaxf(z, 0.0f); }

// The largest value of `values[0..n)` and its index (the lowest index among equals), found by a whole warp.
__device__ __forceinline__ void warp_argmax(const float* values, int n, int lane, float& best, int& where) {
  best = -INFINITY;
  where = INT_MAX;
  for (int i = lane; i < n; i += 32) {
    const float v = values[i];
    if (v > best || (v == best && i < where)) { best = v; where = i; }
  }
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) {
    const float other = __shfl_xor_sync(0xffffffffu, best, offset);
    const int other_where = __shfl_xor_sync(0xffffffffu, where, offset);
    if (other > best || (other == best && other_where < where)) { best = other; where = other_where; }
  }
}

// One warp per token.  Loops over the few outputs stay rolled: in a decode step the weights of a layer pass through the L2
// between two launches, so every line of instructions is fetched from memory again.  Shared memory per warp: 4 arrays of `outputs` floats (scores, choice values, group maxima,
// kept flags).
__global__ void __launch_bounds__(128) router_topk_kernel(const float* __restrict__ logits, long long ld,
                                                          const float* __restrict__ correction, int tokens, int outputs,
                                                          int top, int group_count, int group_keep, int group_pairs,
                                                          int logistic, int over_sum, float factor, int* __restrict__ ids,
                                                          float* __restrict__ weights) {
  extern __shared__ float router_smem[];
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * 4 + warp;
  if (t >= tokens) return;
  float* score = router_smem + (size_t)warp * 4 * outputs;
  float* choice = score + outputs;
  float* group_best = choice + outputs;
  float* kept = group_best + outputs;
  // the correction is the model's: fetched before the logits are there
#pragma unroll 1
  for (int i = lane; i < outputs; i += 32) choice[i] = correction != nullptr ? correction[i] : 0.0f;
  pdl_wait();
  const float* z = logits + (size_t)t * ld;
  if (logistic) {
#pragma unroll 1
    for (int i = lane; i < outputs; i += 32) {
      const float s = 1.0f / (1.0f + expf(-z[i]));
      score[i] = s;
      // the logits order like the scores and do not saturate (sums of two do not order alike)
      choice[i] = correction != nullptr || group_pairs ? s + choice[i] : z[i];
    }
  } else {
    float m = -INFINITY;
    for (int i = lane; i < outputs; i += 32) m = fmaxf(m, z[i]);
    m = warp_max(m);
    float sum = 0.0f;
    for (int i = lane; i < outputs; i += 32) {
      const float e = expf(z[i] - m);
      score[i] = e;
      sum += e;
    }
    sum = warp_sum(sum);
    const float inv = 1.0f / sum;
    for (int i = lane; i < outputs; i += 32) {
      const float s = score[i] * inv;
      score[i] = s;
      choice[i] += s;
    }
  }
  __syncwarp();
  if (group_count > 1 && group_keep < group_count) {
    const int per = outputs / group_count;
    if (per <= 32) {
      // small groups: a lane takes a group; an output stays if fewer than group_keep groups come before its own
#pragma unroll 1
      for (int g = lane; g < group_count; g += 32) {
        float best = -INFINITY, second = -INFINITY;
#pragma unroll 1
        for (int i = 0; i < per; ++i) {
          const float v = choice[g * per + i];
          second = fmaxf(second, fminf(best, v));
          best = fmaxf(best, v);
        }
        group_best[g] = group_pairs && per > 1 ? best + second : best;
      }
      __syncwarp();
#pragma unroll 1
      for (int i = lane; i < outputs; i += 32) {
        const int g = i / per;
        const float own = group_best[g];
        int before = 0;
#pragma unroll 1
        for (int other = 0; other < group_count; ++other) {
          const float v = group_best[other];
          before += v > own || (v == own && other < g);
        }
        if (before >= group_keep) choice[i] = -INFINITY;
      }
    } else {
      for (int g = 0; g < group_count; ++g) {
        float best = -INFINITY, second = -INFINITY;
        for (int i = lane; i < per; i += 32) {
          const float v = choice[g * per + i];
          second = fmaxf(second, fminf(best, v));
          best = fmaxf(best, v);
        }
        if (group_pairs) {
          // the two largest of the group, added (a group of one has only the one)
#pragma unroll
          for (int offset = 16; offset > 0; offset >>= 1) {
            const float other = __shfl_xor_sync(0xffffffffu, best, offset), third = __shfl_xor_sync(0xffffffffu, second, offset);
            second = fmaxf(fminf(best, other), fmaxf(second, third));
            best = fmaxf(best, other);
          }
          if (per > 1) best += second;
        } else {
          best = warp_max(best);
        }
        if (lane == 0) { group_best[g] = best; kept[g] = 0.0f; }
      }
      __syncwarp();
      for (int n = 0; n < group_keep; ++n) {
        float best;
        int where;
        warp_argmax(group_best, group_count, lane, best, where);
        if (lane == 0 && where < group_count) { kept[where] = 1.0f; group_best[where] = -INFINITY; }
        __syncwarp();
      }
      for (int i = lane; i < outputs; i += 32)
        if (kept[i / per] == 0.0f) choice[i] = -INFINITY;
    }
    __syncwarp();
  }
  float chosen_sum = 0.0f;
  if (outputs <= 64) {
    // few outputs: every lane counts how many come before its own; the chosen ones meet in order of their rank
    int* order = reinterpret_cast<int*>(group_best);               // the groups are settled
#pragma unroll 1
    for (int n = lane; n < top; n += 32) order[n] = 0;
    __syncwarp();
#pragma unroll 1
    for (int i = lane; i < outputs; i += 32) {
      const float own = choice[i];
      int before = 0;
#pragma unroll 1
      for (int other = 0; other < outputs; ++other) {
        const float v = choice[other];
        before += v > own || (v == own && other < i);
      }
      if (before < top) order[before] = i;
    }
    __syncwarp();
#pragma unroll 1
    for (int n = 0; n < top; ++n) chosen_sum += score[order[n]];
    chosen_sum = over_sum ? chosen_sum + 1e-20f : 1.0f;
#pragma unroll 1
    for (int n = lane; n < top; n += 32) {
      ids[(size_t)t * top + n] = order[n];
      weights[(size_t)t * top + n] = score[order[n]] / chosen_sum * factor;
    }
    return;
  }
  for (int n = 0; n < top; ++n) {
    float best;
    int where;
    warp_argmax(choice, outputs, lane, best, where);
    if (where >= outputs) where = 0;
    if (lane == 0) {
      ids[(size_t)t * top + n] = where;
      choice[where] = -INFINITY;
    }
    chosen_sum += score[where];
    __syncwarp();
  }
  chosen_sum = over_sum ? chosen_sum + 1e-20f : 1.0f;
  if (lane == 0)
    for (int n = 0; n < top; ++n) weights[(size_t)t * top + n] = score[ids[(size_t)t * top + n]] / chosen_sum * factor;
}

template <typename T>
__global__ void __launch_bounds__(256) activation_kernel(T* __restrict__ rows, long long ld, int count, int width, int kind,
                                                         const float* __restrict__ params) {
  pdl_trigger();
  pdl_wait();
  float a = 0.0f, b = 0.0f;
  if (kind == 1) {
    a = softplus_f(params[0]);
    b = 0.5f + softplus_f(params[1]);
  }
  const long long total = (long long)count * width;
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
    const long long r = idx / width;
    const int c = (int)(idx - r * width);
    T* at = rows + r * ld + c;
    const float z = to_float<T>(*at);
    float y;
    if (kind == 0) {
      const float p = fmaxf(z, 0.0f);
      y = p * p;
    } else {
      y = z > 0.0f ? fmaf(a * z, z, 0.5f * z) : fmaf(b, expm1f(z) - z, 0.5f * z);
    }
    *at = from_float<T>(y);
  }
}

// The same on eight bfloat16 at a time: rows whose width and stride are multiples of 8 and that start on 16 bytes.
__global__ void __launch_bounds__(256) activation_vec_kernel(__nv_bfloat16* __restrict__ rows, long long ld, int count, int width,
                                                             int kind, const float* __restrict__ params) {
  pdl_trigger();
  pdl_wait();
  float a = 0.0f, b = 0.0f;
  if (kind == 1) {
    a = softplus_f(params[0]);
    b = 0.5f + softplus_f(params[1]);
  }
  const int per_row = width / 8;
  const long long total = (long long)count * per_row;
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
    const long long r = idx / per_row;
    const int c = (int)(idx - r * per_row);
    uint4* at = reinterpret_cast<uint4*>(rows + r * ld) + c;
    uint4 raw = *at;
    __nv_bfloat162* two = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float2 z = __bfloat1622float2(two[i]);
      if (kind == 0) {
        const float p = fmaxf(z.x, 0.0f), q = fmaxf(z.y, 0.0f);
        z.x = p * p;
        z.y = q * q;
      } else {
        z.x = z.x > 0.0f ? fmaf(a * z.x, z.x, 0.5f * z.x) : fmaf(b, expm1f(z.x) - z.x, 0.5f * z.x);
        z.y = z.y > 0.0f ? fmaf(a * z.y, z.y, 0.5f * z.y) : fmaf(b, expm1f(z.y) - z.y, 0.5f * z.y);
      }
      two[i] = __floats2bfloat162_rn(z.x, z.y);
    }
    *at = raw;
  }
}

// sum_k a[k] * b[k] over a warp: every lane takes the elements lane, lane + 32, ... in ascending order and the lanes'
// sums meet in a butterfly, so the order depends on nothing but n.
template <typename T>
__device__ __forceinline__ float warp_dot(const T* __restrict__ a, const T* __restrict__ b, int n, int lane) {
  float acc = 0.0f;
  for (int k = lane; k < n; k += 32) acc = fmaf(to_float<T>(a[k]), to_float<T>(b[k]), acc);
  return warp_sum(acc);
}
template <>
__device__ __forceinline__ float warp_dot<__nv_bfloat16>(const __nv_bfloat16* __restrict__ a, const __nv_bfloat16* __restrict__ b,
                                                        int n, int lane) {
  float acc = 0.0f;
  if ((n & 7) == 0 && (((uintptr_t)a | (uintptr_t)b) & 15) == 0) {
    for (int k = lane * 8; k < n; k += 256) {
      const uint4 va = *reinterpret_cast<const uint4*>(a + k), vb = *reinterpret_cast<const uint4*>(b + k);
      const __nv_bfloat162* pa = reinterpret_cast<const __nv_bfloat162*>(&va);
      const __nv_bfloat162* pb = reinterpret_cast<const __nv_bfloat162*>(&vb);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 fa = __bfloat1622float2(pa[i]), fb = __bfloat1622float2(pb[i]);
        acc = fmaf(fa.x, fb.x, acc);
        acc = fmaf(fa.y, fb.y, acc);
      }
    }
  } else {
    for (int k = lane; k < n; k += 32) acc = fmaf(__bfloat162float(a[k]), __bfloat162float(b[k]), acc);
  }
  return warp_sum(acc);
}

// A gate per token on what a kernel adds to (the output of a feed-forward that every token uses): the logistic function of a
// float32 logit found at z[token * ld].  Null: none.
struct RowGate {
  const float* z;
  long long ld;
};
__device__ __forceinline__ float row_gate(const RowGate& gate, int token) {
  return gate.z != nullptr ? 1.0f / (1.0f + expf(-gate.z[(size_t)token * gate.ld])) : 1.0f;
}

// What an expert applies between its matrices: relu(z)^2, or the clamped gate on interleaved (g, u).
struct ExpertAct {
  int gated;
  float limit, alpha, offset;
};

__device__ __forceinline__ float clamped_gate(const ExpertAct& act, float g, float u) {
  g = fminf(g, act.limit);
  u = fminf(fmaxf(u, -act.limit), act.limit);
  return g / (1.0f + expf(-act.alpha * g)) * (u + act.offset);
}

// inner[pair, j] = relu(z_j)^2 or the gate on (z_2j, z_2j+1), z = w_up[expert] h[token] (times the pair's weight, if the
// weight is the input's), for the pairs whose choice is an expert.
template <typename T>
__global__ void __launch_bounds__(256) expert_up_kernel(const T* __restrict__ h, long long ld_h, const T* __restrict__ w_up,
                                                        const int* __restrict__ ids, const float* __restrict__ in_weights,
                                                        T* __restrict__ inner, int top, int experts, int width, int ff,
                                                        ExpertAct act) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x;
  const int expert = ids[pair];
  if (expert < 0 || expert >= experts) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* row = h + (size_t)(pair / top) * ld_h;
  const float scale = in_weights != nullptr ? in_weights[pair] : 1.0f;
  const T* w = w_up + (size_t)expert * (act.gated ? 2 : 1) * ff * width;
  for (int j = blockIdx.y * 8 + warp; j < ff; j += gridDim.y * 8) {
    if (act.gated) {
      const float g = warp_dot<T>(row, w + (size_t)2 * j * width, width, lane) * scale;
      const float u = warp_dot<T>(row, w + ((size_t)2 * j + 1) * width, width, lane) * scale;
      if (lane == 0) inner[(size_t)pair * ff + j] = from_float<T>(clamped_gate(act, g, u));
      continue;
    }
    const float dot = warp_dot<T>(row, w + (size_t)j * width, width, lane);
    if (lane == 0) {
      const float p = fmaxf(dot * scale, 0.0f);
      inner[(size_t)pair * ff + j] = from_float<T>(p * p);
    }
  }
}

// x[token, n] <- gate * x[token, n] + sum over the token's choices, in their order, of weight * (w_down[expert][n, :] .
// inner[pair, :]), or weight * h[token, n] for an identity expert; null weights and a null gate count as one.
template <typename T>
__global__ void __launch_bounds__(256) expert_down_add_kernel(const T* __restrict__ inner, const T* __restrict__ w_down,
                                                              const T* __restrict__ h, long long ld_h,
                                                              const int* __restrict__ ids, const float* __restrict__ weights,
                                                              float* __restrict__ x, int top, int experts, int width, int ff,
                                                              long long down_expert, long long down_row, RowGate gate) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const float g = row_gate(gate, t);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int n = blockIdx.y * 8 + warp; n < width; n += gridDim.y * 8) {
    float acc = 0.0f;
    for (int k = 0; k < top; ++k) {
      const int pair = t * top + k;
      const int expert = ids[pair];
      const float weight = weights != nullptr ? weights[pair] : 1.0f;
      if (expert >= 0 && expert < experts)
        acc = fmaf(weight, warp_dot<T>(inner + (size_t)pair * ff, w_down + (size_t)expert * down_expert + (size_t)n * down_row, ff, lane), acc);
      else
        acc = fmaf(weight, to_float<T>(h[(size_t)t * ld_h + n]), acc);
    }
    if (lane == 0) x[(size_t)t * width + n] = fmaf(g, x[(size_t)t * width + n], acc);
  }
}

// One block.  place[pair]: the pair's row in the buffer grouped by expert (-1 for an identity expert);
// offsets[e] .. offsets[e + 1]: expert e's rows.
__global__ void __launch_bounds__(1024) expert_sort_kernel(const int* __restrict__ ids, int pairs, int experts,
                                                           int* __restrict__ place, int* __restrict__ offsets) {
  extern __shared__ int sort_smem[];
  int* count = sort_smem;
  int* cursor = sort_smem + experts;
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e < experts; e += blockDim.x) count[e] = 0;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    const int e = ids[p];
    if (e >= 0 && e < experts) atomicAdd(&count[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int running = 0;
    for (int e = 0; e < experts; ++e) {
      offsets[e] = running;
      cursor[e] = running;
      running += count[e];
    }
    offsets[experts] = running;
  }
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    const int e = ids[p];
    place[p] = (e >= 0 && e < experts) ? atomicAdd(&cursor[e], 1) : -1;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) expert_gather_kernel(const T* __restrict__ h, long long ld_h, const int* __restrict__ place,
                                                            const float* __restrict__ in_weights, T* __restrict__ grouped,
                                                            int top, int width) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x;
  const int row = place[pair];
  if (row < 0) return;
  const T* src = h + (size_t)(pair / top) * ld_h;
  T* dst = grouped + (size_t)row * width;
  const float scale = in_weights != nullptr ? in_weights[pair] : 1.0f;
  if (sizeof(T) == 2 && width % 8 == 0 && ld_h % 8 == 0 && ((uintptr_t)h & 15) == 0 && ((uintptr_t)grouped & 15) == 0) {
    for (int i = threadIdx.x; i < width / 8; i += blockDim.x) {
      uint4 raw = reinterpret_cast<const uint4*>(src)[i];
      if (in_weights != nullptr) {
        __nv_bfloat162* two = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = __bfloat1622float2(two[e]);
          two[e] = __floats2bfloat162_rn(f.x * scale, f.y * scale);
        }
      }
      reinterpret_cast<uint4*>(dst)[i] = raw;
    }
    return;
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x)
    dst[i] = in_weights != nullptr ? from_float<T>(to_float<T>(src[i]) * scale) : src[i];
}

template <typename T>
__global__ void __launch_bounds__(256) expert_combine_add_kernel(const float* __restrict__ outputs, const int* __restrict__ place,
                                                                 const float* __restrict__ weights, const T* __restrict__ h,
                                                                 long long ld_h, float* __restrict__ x, int top, int width,
                                                                 RowGate gate) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const float g = row_gate(gate, t);
  for (int n = blockIdx.y * blockDim.x + threadIdx.x; n < width; n += gridDim.y * blockDim.x) {
    float acc = 0.0f;
    for (int k = 0; k < top; ++k) {
      const int pair = t * top + k;
      const int row = place[pair];
      const float v = row >= 0 ? outputs[(size_t)row * width + n] : to_float<T>(h[(size_t)t * ld_h + n]);
      acc = fmaf(weights != nullptr ? weights[pair] : 1.0f, v, acc);
    }
    x[(size_t)t * width + n] = fmaf(g, x[(size_t)t * width + n], acc);
  }
}

// The dense path, between its two products.  z [tokens, experts * ff]: every expert's up projection of every token.
// In place: a token's rows of a chosen expert become weight * relu(z)^2, all others zero, so that ONE product with
// the down matrices side by side along k adds the weighted sum of the chosen experts.  Blocks with blockIdx.y ==
// experts add the identity experts' share, weight * h, into the stream.
template <typename T>
__global__ void __launch_bounds__(256) expert_dense_weigh_kernel(T* __restrict__ z, const int* __restrict__ ids,
                                                                 const float* __restrict__ weights, const T* __restrict__ h,
                                                                 long long ld_h, float* __restrict__ x, int top, int experts,
                                                                 int width, int ff) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, e = blockIdx.y;
  if (e == experts) {
    float w = 0.0f;
    bool any = false;
    for (int k = 0; k < top; ++k) {
      const int id = ids[t * top + k];
      if (id >= experts) { w += weights[t * top + k]; any = true; }
    }
    if (!any) return;
    for (int n = threadIdx.x; n < width; n += blockDim.x) x[(size_t)t * width + n] += w * to_float<T>(h[(size_t)t * ld_h + n]);
    return;
  }
  float w = 0.0f;
  bool chosen = false;
  for (int k = 0; k < top; ++k)
    if (ids[t * top + k] == e) { w = weights[t * top + k]; chosen = true; }
  T* row = z + ((size_t)t * experts + e) * ff;
  if (!chosen) {
    for (int j = threadIdx.x; j < ff; j += blockDim.x) row[j] = from_float<T>(0.0f);
    return;
  }
  for (int j = threadIdx.x; j < ff; j += blockDim.x) {
    const float p = fmaxf(to_float<T>(row[j]), 0.0f);
    row[j] = from_float<T>(w * p * p);
  }
}

// The dense path of gated experts: z [tokens, experts * 2 ff] (interleaved gate and up of every expert) -> out [tokens,
// experts * ff], a chosen expert's activated values and zeros elsewhere.  `weigh_input`: the weight multiplies (g, u), else
// the activated value.  `shared_ff` > 0: behind the experts' columns lie those of a feed-forward that every token uses
// (2 shared_ff in z, shared_ff in out), its activated values times the token's gate; blocks with blockIdx.y == experts do it.
template <typename T>
__global__ void __launch_bounds__(256) expert_dense_gate_kernel(const T* __restrict__ z, const int* __restrict__ ids,
                                                                const float* __restrict__ weights, T* __restrict__ out, int top,
                                                                int experts, int expert_ff, int weigh_input, ExpertAct act,
                                                                int shared_ff, RowGate gate) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, e = blockIdx.y;
  float w = 0.0f;
  bool chosen = false;
  if (e == experts) {
    w = row_gate(gate, t);
    chosen = true;
    weigh_input = 0;
  } else {
    for (int k = 0; k < top; ++k)
      if (ids[t * top + k] == e) { w = weights[t * top + k]; chosen = true; }
  }
  const size_t row = (size_t)experts * expert_ff + shared_ff;
  const int ff = e == experts ? shared_ff : expert_ff;
  const T* src = z + ((size_t)t * row + (size_t)e * expert_ff) * 2;
  T* dst = out + (size_t)t * row + (size_t)e * expert_ff;
  const float in = weigh_input ? w : 1.0f, after = weigh_input ? 1.0f : w;
  if (sizeof(T) == 2 && expert_ff % 4 == 0 && shared_ff % 4 == 0) {
    // four values at a time: 16 bytes in, 8 bytes out (the buffers are the wrapper's own, so aligned)
    for (int j = threadIdx.x; j < ff / 4; j += blockDim.x) {
      uint2 packed = make_uint2(0u, 0u);
      if (chosen) {
        const uint4 raw = reinterpret_cast<const uint4*>(src)[j];
        const __nv_bfloat162* two = reinterpret_cast<const __nv_bfloat162*>(&raw);
        float y[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 gu = __bfloat1622float2(two[i]);
          y[i] = after * clamped_gate(act, gu.x * in, gu.y * in);
        }
        *reinterpret_cast<__nv_bfloat162*>(&packed.x) = __floats2bfloat162_rn(y[0], y[1]);
        *reinterpret_cast<__nv_bfloat162*>(&packed.y) = __floats2bfloat162_rn(y[2], y[3]);
      }
      reinterpret_cast<uint2*>(dst)[j] = packed;
    }
    return;
  }
  for (int j = threadIdx.x; j < ff; j += blockDim.x)
    dst[j] = from_float<T>(chosen ? after * clamped_gate(act, to_float<T>(src[2 * j]) * in, to_float<T>(src[2 * j + 1]) * in) : 0.0f);
}

}  // namespace

// logits float32 [tokens, ld]; correction float32 [outputs] or null; ids int32 [tokens, top]; weights float32 [tokens, top].
TGE_API int tge_router_topk(const float* logits, long long ld, const float* correction, int tokens, int outputs, int top,
                            int group_count, int group_keep, int group_pairs, int logistic, int over_sum, float factor,
                            int* ids, float* weights, cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && outputs > 0 && outputs <= 1024, "router_topk: 1 to 1024 outputs, not %d", outputs);
  TGE_REQUIRE(top > 0 && top <= outputs, "router_topk: %d choices of %d outputs", top, outputs);
  TGE_REQUIRE(group_count > 0 && outputs % group_count == 0 && group_keep > 0 && group_keep <= group_count,
              "router_topk: %d groups (%d kept) of %d outputs", group_count, group_keep, outputs);
  TGE_REQUIRE((outputs / group_count) * group_keep >= top, "router_topk: %d choices do not fit the kept groups", top);
  if (tokens == 0) return 0;
  const size_t smem = (size_t)4 * 4 * outputs * sizeof(float);
  if (smem > 48 * 1024) {
    static bool configured = false;
    if (!configured) {
      cudaFuncSetAttribute(router_topk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 4 * 4 * 1024 * (int)sizeof(float));
      configured = true;
    }
  }
  tge_launch(router_topk_kernel, dim3((tokens + 3) / 4), dim3(128), smem, stream, logits, ld, correction, tokens, outputs, top,
             group_count, group_keep, group_pairs, logistic, over_sum, factor, ids, weights);
  return tge_launched("router_topk", 1);
}

// rows: run dtype [count, width] with row stride ld, changed in place.  kind 0: relu(z)^2; 1: the two-parameter form,
// params float32 [2] on the device.
TGE_API int tge_activation(void* rows, long long ld, int count, int width, int kind, const float* params, int is_bf16,
                           cudaStream_t stream) {
  TGE_REQUIRE(count >= 0 && width > 0 && ld >= width, "activation: bad shape");
  TGE_REQUIRE(kind == 0 || (kind == 1 && params != nullptr), "activation: kind %d", kind);
  if (count == 0) return 0;
  const long long total = (long long)count * width;
  if (is_bf16 && width % 8 == 0 && ld % 8 == 0 && (uintptr_t)rows % 16 == 0) {
    const long long vectors = total / 8;
    const int vec_blocks = (int)((vectors + 255) / 256 > 148 * 32 ? 148 * 32 : (vectors + 255) / 256);
    tge_launch(activation_vec_kernel, dim3(vec_blocks), dim3(256), 0, stream, (__nv_bfloat16*)rows, ld, count, width, kind, params);
    return tge_launched("activation", 1);
  }
  const int blocks = (int)((total + 255) / 256 > 148 * 32 ? 148 * 32 : (total + 255) / 256);
  if (is_bf16) tge_launch(activation_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (__nv_bfloat16*)rows, ld, count, width, kind, params);
  else tge_launch(activation_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)rows, ld, count, width, kind, params);
  return tge_launched("activation", 1);
}

// The direct path.  h: run dtype [tokens, >= width] with row stride ld_h; w_up [experts, ff, width]; row n of expert
// e's down matrix (ff numbers) starts at w_down + e * down_expert + n * down_row; inner: run dtype scratch
// [tokens * top, ff]; x: the float32 stream [tokens, width].  With `gated` w_up is [experts, 2 ff, width], gate and up rows
// interleaved.
TGE_API int tge_experts_direct(const void* h, long long ld_h, const void* w_up, const void* w_down, long long down_expert,
                               long long down_row, const int* ids, const float* weights, void* inner, float* x, int tokens,
                               int top, int experts, int width, int ff, int weigh_input, int gated, float limit,
                               float alpha, float offset, const float* x_gate, long long ld_gate, int is_bf16,
                               cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && top > 0 && experts >= 0 && width > 0 && ff > 0, "experts: bad shape");
  TGE_REQUIRE(!gated || limit > 0.0f, "experts: the gate's limit must be positive");
  if (tokens == 0) return 0;
  const ExpertAct act{gated, limit, alpha, offset};
  const RowGate gate{x_gate, ld_gate};
  const float* in_weights = weigh_input ? weights : nullptr;
  if (weigh_input) weights = nullptr;
  const int up_y = (ff + 7) / 8 < 64 ? (ff + 7) / 8 : 64;
  const int down_y = (width + 7) / 8 < 64 ? (width + 7) / 8 : 64;
  if (is_bf16) {
    tge_launch(expert_up_kernel<__nv_bfloat16>, dim3(tokens * top, up_y), dim3(256), 0, stream, (const __nv_bfloat16*)h, ld_h,
               (const __nv_bfloat16*)w_up, ids, in_weights, (__nv_bfloat16*)inner, top, experts, width, ff, act);
    tge_launch(expert_down_add_kernel<__nv_bfloat16>, dim3(tokens, down_y), dim3(256), 0, stream, (const __nv_bfloat16*)inner,
               (const __nv_bfloat16*)w_down, (const __nv_bfloat16*)h, ld_h, ids, weights, x, top, experts, width, ff, down_expert,
               down_row, gate);
  } else {
    tge_launch(expert_up_kernel<float>, dim3(tokens * top, up_y), dim3(256), 0, stream, (const float*)h, ld_h,
               (const float*)w_up, ids, in_weights, (float*)inner, top, experts, width, ff, act);
    tge_launch(expert_down_add_kernel<float>, dim3(tokens, down_y), dim3(256), 0, stream, (const float*)inner,
               (const float*)w_down, (const float*)h, ld_h, ids, weights, x, top, experts, width, ff, down_expert, down_row,
               gate);
  }
  return tge_launched("experts_direct", 2);
}

// The grouped path, first half: place int32 [tokens * top], offsets int32 [experts + 1], grouped run dtype
// [tokens * top, width] (the rows of expert e at offsets[e] .. offsets[e + 1]), times the pairs' weights if given.
TGE_API int tge_experts_group(const void* h, long long ld_h, const int* ids, const float* in_weights, int* place, int* offsets,
                              void* grouped, int tokens, int top, int experts, int width, int is_bf16, cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && top > 0 && experts > 0 && experts <= 4096 && width > 0, "experts: bad shape");
  if (tokens == 0) return 0;
  tge_launch(expert_sort_kernel, dim3(1), dim3(1024), (size_t)2 * experts * sizeof(int), stream, ids, tokens * top, experts,
             place, offsets);
  if (is_bf16)
    tge_launch(expert_gather_kernel<__nv_bfloat16>, dim3(tokens * top), dim3(256), 0, stream, (const __nv_bfloat16*)h, ld_h,
               (const int*)place, in_weights, (__nv_bfloat16*)grouped, top, width);
  else
    tge_launch(expert_gather_kernel<float>, dim3(tokens * top), dim3(256), 0, stream, (const float*)h, ld_h, (const int*)place,
               in_weights, (float*)grouped, top, width);
  return tge_launched("experts_group", 2);
}

// The grouped path, second half: outputs float32 [tokens * top, width] in grouped order.
TGE_API int tge_experts_combine_add(const float* outputs, const int* place, const float* weights, const void* h, long long ld_h,
                                    float* x, int tokens, int top, int width, const float* x_gate, long long ld_gate,
                                    int is_bf16, cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && top > 0 && width > 0, "experts: bad shape");
  if (tokens == 0) return 0;
  const RowGate gate{x_gate, ld_gate};
  const int chunks = (width + 1023) / 1024;
  if (is_bf16)
    tge_launch(expert_combine_add_kernel<__nv_bfloat16>, dim3(tokens, chunks), dim3(256), 0, stream, outputs, place, weights,
               (const __nv_bfloat16*)h, ld_h, x, top, width, gate);
  else
    tge_launch(expert_combine_add_kernel<float>, dim3(tokens, chunks), dim3(256), 0, stream, outputs, place, weights,
               (const float*)h, ld_h, x, top, width, gate);
  return tge_launched("experts_combine_add", 1);
}

// The dense path: z run dtype [tokens, experts * ff] in place (see the kernel); x float32 [tokens, width].
TGE_API int tge_experts_dense_weigh(void* z, const int* ids, const float* weights, const void* h, long long ld_h, float* x,
                                    int tokens, int top, int experts, int width, int ff, int is_bf16, cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && top > 0 && experts > 0 && experts < 65535 && width > 0 && ff > 0, "experts: bad shape");
  if (tokens == 0) return 0;
  if (is_bf16)
    tge_launch(expert_dense_weigh_kernel<__nv_bfloat16>, dim3(tokens, experts + 1), dim3(256), 0, stream, (__nv_bfloat16*)z, ids,
               weights, (const __nv_bfloat16*)h, ld_h, x, top, experts, width, ff);
  else
    tge_launch(expert_dense_weigh_kernel<float>, dim3(tokens, experts + 1), dim3(256), 0, stream, (float*)z, ids, weights,
               (const float*)h, ld_h, x, top, experts, width, ff);
  return tge_launched("experts_dense_weigh", 1);
}

// The dense path of gated experts: z run dtype [tokens, 2 (experts * ff + shared_ff)] -> out [tokens, experts * ff +
// shared_ff] (see the kernel).
TGE_API int tge_experts_dense_gate(const void* z, const int* ids, const float* weights, void* out, int tokens, int top,
                                   int experts, int ff, int weigh_input, float limit, float alpha, float offset, int shared_ff,
                                   const float* shared_gate, long long ld_gate, int is_bf16, cudaStream_t stream) {
  TGE_REQUIRE(tokens >= 0 && top > 0 && experts > 0 && experts < 65535 && ff > 0 && shared_ff >= 0 && limit > 0.0f, "experts: bad shape");
  TGE_REQUIRE(((uintptr_t)z & 15) == 0 && ((uintptr_t)out & 15) == 0, "experts: rows must start on 16 bytes");
  if (tokens == 0) return 0;
  const ExpertAct act{1, limit, alpha, offset};
  const RowGate gate{shared_gate, ld_gate};
  const dim3 grid(tokens, experts + (shared_ff > 0 ? 1 : 0));
  if (is_bf16)
    tge_launch(expert_dense_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)z, ids,
               weights, (__nv_bfloat16*)out, top, experts, ff, weigh_input, act, shared_ff, gate);
  else
    tge_launch(expert_dense_gate_kernel<float>, grid, dim3(256), 0, stream, (const float*)z, ids, weights,
               (float*)out, top, experts, ff, weigh_input, act, shared_ff, gate);
  return tge_launched("experts_dense_gate", 1);
}
