// Learned absolute positions and the post-norm residual.
//   embed_positions_kernel   x[t] = table[token] + pos_table[position]; also the act-dtype copy the first sublayer reads
//   postnorm_add_kernel      x[t] += rms_norm(y[t]) * w, where y is a sublayer's output: the sublayer read x itself, and
//                            its output passes through the norm on its way INTO the residual.  y is either a plain row or
//                            gathered here from a mixture of experts (weighted rows of the grouped down projection plus
//                            the gated shared expert), so the mixture's sum never goes through memory.
//   sum_norm_kernel          x[t] = rms_norm(alpha x[t] + y[t]) * w: the norm's output REPLACES the residual (y plain or a
//                            mixture, in which a negative row number stands for x[t] itself)
//   embed_pairs_kernel       x[t] = table[token] * scale + pairs[hash(previous token, token)]
// One CTA per token row; the row of y stays in shared memory between the two passes.
#include "hyb_common.cuh"

namespace pieh {

template <typename ET, typename AT>
__global__ void embed_positions_kernel(float* x, AT* act, const ET* table, const ET* pos_table, const int32_t* tokens,
                                       const int32_t* positions, int W, int vocab, int max_pos) {
  pdl_sync();
  const int t = blockIdx.x;
  int id = tokens[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const ET* row = table + (size_t)id * W;
  const ET* prow = nullptr;
  if (pos_table) {
    int p = positions[t];
    p = p < 0 ? 0 : (p >= max_pos ? max_pos - 1 : p);
    prow = pos_table + (size_t)p * W;
  }
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float v = elem<ET>::load(row + c);
    if (prow) v += elem<ET>::load(prow + c);
    x[(size_t)t * W + c] = v;
    if (act) elem<AT>::store(act + (size_t)t * W + c, v);
  }
}

template <typename AT>
__global__ void __launch_bounds__(256) postnorm_add_kernel(float* x, AT* act, const float* y, const pieh_mix_sum mix,
                                                           const float* norm_w, float eps, int W) {
  extern __shared__ float row[];
  __shared__ float red[33];
  pdl_sync();
  const int t = blockIdx.x;
  float ss = 0.f;
  if (mix.parts) {
    float sg = 0.f;
    if (mix.shared) sg = 1.f / (1.f + expf(-mix.shared_gate[(size_t)t * mix.gate_ld]));
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      float v = 0.f;
      for (int k = 0; k < mix.top; ++k)   // fixed order: the sum does not depend on how the slots were handed out
        v = fmaf(mix.part_w[(size_t)t * mix.top + k], mix.parts[(size_t)mix.part_row[(size_t)t * mix.top + k] * W + c], v);
      if (mix.shared) v = fmaf(sg, mix.shared[(size_t)t * W + c], v);
      row[c] = v;
      ss = fmaf(v, v, ss);
    }
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
      const float v = y[(size_t)t * W + c];
      row[c] = v;
      ss = fmaf(v, v, ss);
    }
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)W + eps);
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float v = x[(size_t)t * W + c] + row[c] * inv * norm_w[c];
    x[(size_t)t * W + c] = v;
    if (act) elem<AT>::store(act + (size_t)t * W + c, v);
  }
}

template <typename AT, int V> struct act_run;   // V consecutive act elements
template <> struct act_run<float, 1> { static __device__ __forceinline__ void store(float* p, const float* v) { *p = v[0]; } };
template <> struct act_run<__nv_bfloat16, 1> {
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct act_run<float, 4> {
  static __device__ __forceinline__ void store(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct act_run<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  }
};
template <int V> __device__ __forceinline__ void load_run(const float* p, float (&v)[V]) {
  if (V == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1 % V] = x.y; v[2 % V] = x.z; v[3 % V] = x.w;
  } else v[0] = *p;
}

constexpr int kMaxMix = 32;

// V = 4: W a multiple of 4 and every row 16-byte aligned
template <typename AT, int V>
__global__ void __launch_bounds__(256) sum_norm_kernel(float* x, AT* act, const float* y, const pieh_mix_sum mix,
                                                       const float* norm_w, float alpha, float eps, int W) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[33], pw[kMaxMix];
  __shared__ int pr[kMaxMix];
  pdl_sync();
  const int t = blockIdx.x;
  float keep = alpha;          // what multiplies x: alpha plus the weights of the identity experts
  int top = 0;
  float sg = 1.f;
  if (mix.parts) {
    top = mix.top;
    for (int k = threadIdx.x; k < top; k += blockDim.x) {
      pr[k] = mix.part_row[(size_t)t * top + k];
      pw[k] = mix.part_w[(size_t)t * top + k];
    }
    if (mix.shared && mix.shared_gate) sg = 1.f / (1.f + expf(-mix.shared_gate[(size_t)t * mix.gate_ld]));
    __syncthreads();
    for (int k = 0; k < top; ++k)
      if (pr[k] < 0) keep += pw[k];
  }
  float ss = 0.f;
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
    float v[V], u[V];
    load_run<V>(x + (size_t)t * W + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= keep;
    if (mix.parts) {
      for (int k = 0; k < top; ++k) {   // choice order: the sum does not depend on how the slots were handed out
        if (pr[k] < 0) continue;
        load_run<V>(mix.parts + (size_t)pr[k] * W + c, u);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = fmaf(pw[k], u[e], v[e]);
      }
      if (mix.shared) {
        load_run<V>(mix.shared + (size_t)t * W + c, u);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = fmaf(sg, u[e], v[e]);
      }
    } else {
      load_run<V>(y + (size_t)t * W + c, u);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += u[e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
    act_run<float, V>::store(row + c, v);
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)W + eps);
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {   // each thread reads back the entries it wrote
    float v[V], w[V];
    load_run<V>(row + c, v);
    load_run<V>(norm_w + c, w);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] *= inv * w[e];
    act_run<float, V>::store(x + (size_t)t * W + c, v);
    if (act) act_run<AT, V>::store(act + (size_t)t * W + c, v);
  }
}

template <typename ET, typename AT>
__global__ void embed_pairs_kernel(float* x, AT* act, const ET* table, const ET* pairs, const int32_t* tokens, float scale,
                                   long long mul_prev, long long mul_cur, int buckets, int32_t* prev, int W, int vocab,
                                   const pieh_batch b) {
  __shared__ int prow;
  pdl_sync();
  const int t = blockIdx.x;
  const int i = b.tok_seq[t], start = b.seq_start[i];
  int id = tokens[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  if (pairs && threadIdx.x == 0) {
    long long before = -1;
    if (t > start) before = tokens[t - 1];
    else {
      // this row alone reads the stored token, so it is also the one that moves it on to the portion's last token
      int32_t* mine = prev + b.seq_slot[i];
      if (b.seq_ctx[i] > 0) before = *mine;
      *mine = tokens[start + b.seq_len[i] - 1];
    }
    long long r = buckets;
    if (before >= 0) {
      r = (before * mul_prev + tokens[t] * mul_cur) % buckets;
      if (r < 0) r += buckets;
    }
    prow = (int)r;
  }
  __syncthreads();
  const ET* row = table + (size_t)id * W;
  const ET* pr = pairs ? pairs + (size_t)prow * W : nullptr;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float v = elem<ET>::load(row + c) * scale;
    if (pr) v += elem<ET>::load(pr + c);
    x[(size_t)t * W + c] = v;
    if (act) elem<AT>::store(act + (size_t)t * W + c, v);
  }
}

}  // namespace pieh

using namespace pieh;

extern "C" int pieh_embed_positions(float* x, void* act, int act_dtype, const void* table, const void* pos_table,
                                    int table_dtype, const int32_t* tokens, const int32_t* positions, int T, int W, int vocab,
                                    int max_positions, void* stream) {
  if (!x || !table || !tokens || (pos_table && !positions)) return PIE_ENULL;
  if (T < 0 || W < 1 || vocab < 1 || (pos_table && max_positions < 1)) return PIE_EINVAL_SHAPE;
  if (T == 0) return PIE_OK;
  cudaStream_t st = (cudaStream_t)stream;
  count_launch();
  PIEH_DISPATCH_DTYPE(table_dtype, ET, PIEH_DISPATCH_DTYPE(act_dtype, AT,
      launch_k(embed_positions_kernel<ET, AT>, dim3(T), dim3(256), 0, st, x, (AT*)act, (const ET*)table, (const ET*)pos_table,
               tokens, positions, W, vocab, max_positions)));
  return status_of(cudaGetLastError());
}

extern "C" int pieh_postnorm_add(float* x, void* act, int act_dtype, const float* y, const pieh_mix_sum* mix,
                                 const float* norm_w, float eps, int T, int W, void* stream) {
  if (!x || !norm_w || (!y && !(mix && mix->parts))) return PIE_ENULL;
  if (mix && mix->parts && (!mix->part_row || !mix->part_w || mix->top < 1 || (mix->shared && !mix->shared_gate)))
    return PIE_ENULL;
  if (T < 0 || W < 1 || (size_t)W * 4 > 200 * 1024) return PIE_EINVAL_SHAPE;
  if (T == 0) return PIE_OK;
  cudaStream_t st = (cudaStream_t)stream;
  pieh_mix_sum m = {};
  if (mix && mix->parts) m = *mix;
  const size_t smem = (size_t)W * 4;
  if (smem > 48 * 1024) {
    cudaFuncSetAttribute(postnorm_add_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaFuncSetAttribute(postnorm_add_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  }
  count_launch();
  PIEH_DISPATCH_DTYPE(act_dtype, AT, launch_k(postnorm_add_kernel<AT>, dim3(T), dim3(256), smem, st, x, (AT*)act, y, m, norm_w, eps, W));
  return status_of(cudaGetLastError());
}

extern "C" int pieh_sum_norm(float* x, void* act, int act_dtype, const float* y, const pieh_mix_sum* mix,
                             const float* norm_w, float alpha, float eps, int T, int W, void* stream) {
  const bool has_mix = mix && mix->parts;
  if (!x || !norm_w || (!y && !has_mix)) return PIE_ENULL;
  if (has_mix && (!mix->part_row || !mix->part_w)) return PIE_ENULL;
  if (T < 0 || W < 1 || (size_t)W * 4 > 200 * 1024 || (has_mix && (mix->top < 1 || mix->top > kMaxMix))) return PIE_EINVAL_SHAPE;
  if (T == 0) return PIE_OK;
  pieh_mix_sum m = {};
  if (has_mix) m = *mix;
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = W % 4 == 0 && al(x) && al(act) && al(y) && al(norm_w) && al(m.parts) && al(m.shared);
  const size_t smem = (size_t)W * 4;
  count_launch();
  cudaError_t e = cudaSuccess;
  PIEH_DISPATCH_DTYPE(act_dtype, AT, {
    auto kernel = vec ? sum_norm_kernel<AT, 4> : sum_norm_kernel<AT, 1>;
    if (smem > 48 * 1024) e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = launch_k(kernel, dim3(T), dim3(256), smem, (cudaStream_t)stream, x, (AT*)act, y, m, norm_w, alpha, eps, W);
  });
  return status_of(e);
}

extern "C" int pieh_embed_pairs(float* x, void* act, int act_dtype, const void* table, const void* pairs, int table_dtype,
                                const int32_t* tokens, float scale, long long mul_prev, long long mul_cur, int buckets, int32_t* prev, int W,
                                int vocab, const pieh_batch* b, void* stream) {
  if (!x || !table || !tokens || !b || (pairs && !prev)) return PIE_ENULL;
  if (W < 1 || vocab < 1 || (pairs && buckets < 1)) return PIE_EINVAL_SHAPE;
  if (b->T == 0) return PIE_OK;
  count_launch();
  cudaError_t e = cudaSuccess;
  PIEH_DISPATCH_DTYPE(table_dtype, ET, PIEH_DISPATCH_DTYPE(act_dtype, AT,
      e = launch_k(embed_pairs_kernel<ET, AT>, dim3(b->T), dim3(256), 0, (cudaStream_t)stream, x, (AT*)act, (const ET*)table,
                   (const ET*)pairs, tokens, scale, mul_prev, mul_cur, buckets, prev, W, vocab, *b)));
  return status_of(e);
}
