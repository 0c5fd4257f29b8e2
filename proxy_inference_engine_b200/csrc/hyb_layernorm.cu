// Sandwich blocks built on layer norm (mean taken off, weight and bias).
//   layernorm_add_kernel   x[t] += ln(y[t]) * post_w + post_b -- or x[t] = y[t] -- plus an optional saved row and a vector; then
//                          h = ln(x[t]) * next_w + next_b (or x[t] itself) in the act dtype: the norm on a sublayer's output, the
//                          residual sum and the next sublayer's norm are ONE pass over the residual.  With a row list only the
//                          listed rows are formed and x stays as it is (the model's final norm).
// One CTA per row, the row in registers (16-byte accesses); a variance is the mean of the squared deviations from the mean
// already found (two reductions, no cancellation).  Every sum has a fixed order, so a row does not depend on what else runs.
#include "hyb_common.cuh"

namespace pieh {

struct LnAdd {
  float* x;
  const float* y; long long y_ld;
  const float* post_w; const float* post_b;
  const float* add_rows; long long add_ld;
  const float* add_vec;
  void* h;
  const float* next_w; const float* next_b;
  const int32_t* rows;
  float eps;
  int W;
};

// sum over the CTA (at most 8 warps); each call of a kernel brings its own `red`, so one barrier is enough
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) s += red[w];
  return s;
}

__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}
__device__ __forceinline__ float4 get4(const float* p) { return *reinterpret_cast<const float4*>(p); }

// v <- (v - mean(v)) / sqrt(mean((v - mean)^2) + eps) * w + b, the row spread over the CTA's registers
template <int NV>
__device__ __forceinline__ void ln_rows(float4 (&v)[NV], const float* w, const float* b, float eps, int W, float* red) {
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);   // what lies past the row is zero
  const float mean = cta_sum(s, red) / (float)W;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    if ((int)(threadIdx.x + i * blockDim.x) * 4 < W) {
      v[i].x -= mean; v[i].y -= mean; v[i].z -= mean; v[i].w -= mean;
      q = fmaf(v[i].x, v[i].x, q); q = fmaf(v[i].y, v[i].y, q); q = fmaf(v[i].z, v[i].z, q); q = fmaf(v[i].w, v[i].w, q);
    }
  }
  const float inv = 1.f / sqrtf(cta_sum(q, red + 8) / (float)W + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < W) {
      const float4 g = get4(w + c), o = get4(b + c);
      v[i].x = fmaf(v[i].x * inv, g.x, o.x); v[i].y = fmaf(v[i].y * inv, g.y, o.y);
      v[i].z = fmaf(v[i].z * inv, g.z, o.z); v[i].w = fmaf(v[i].w * inv, g.w, o.w);
    }
  }
}

template <typename AT, int NV>   // NV runs of 4 elements a thread
__global__ void __launch_bounds__(256) layernorm_add_kernel(const LnAdd a) {
  __shared__ float red[4][8];
  pdl_sync();
  const int W = a.W;
  const int t = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  float* xr = a.x + (size_t)t * W;
  const float* yr = a.y ? a.y + (size_t)t * a.y_ld : nullptr;
  const bool replace = yr && !a.post_w;
  float4 v[NV], u[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {   // both rows are on their way before the first reduction
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    v[i] = u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < W) {
      if (replace) v[i] = get4(yr + c);
      else {
        v[i] = get4(xr + c);
        if (yr) u[i] = get4(yr + c);
      }
    }
  }
  if (yr && !replace) ln_rows<NV>(u, a.post_w, a.post_b, a.eps, W, red[0]);
  const bool changed = yr || a.add_rows || a.add_vec;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c >= W) continue;
    v[i].x += u[i].x; v[i].y += u[i].y; v[i].z += u[i].z; v[i].w += u[i].w;
    if (a.add_rows) {
      const float4 z = get4(a.add_rows + (size_t)t * a.add_ld + c);
      v[i].x += z.x; v[i].y += z.y; v[i].z += z.z; v[i].w += z.w;
    }
    if (a.add_vec) {
      const float4 z = get4(a.add_vec + c);
      v[i].x += z.x; v[i].y += z.y; v[i].z += z.z; v[i].w += z.w;
    }
    if (changed && !a.rows) put4(xr + c, v[i]);
  }
  if (!a.h) return;
  if (a.next_w) ln_rows<NV>(v, a.next_w, a.next_b, a.eps, W, red[2]);
  AT* hr = reinterpret_cast<AT*>(a.h) + (size_t)blockIdx.x * W;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < W) put4(hr + c, v[i]);
  }
}

// any width: the row in shared memory, one element at a time
__device__ __forceinline__ void ln_shared(float* row, const float* w, const float* b, float eps, int W, float* red) {
  float s = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) s += row[c];
  const float mean = cta_sum(s, red) / (float)W;
  float q = 0.f;
  for (int c = threadIdx.x; c < W; c += blockDim.x) { const float d = row[c] - mean; q = fmaf(d, d, q); }
  const float inv = 1.f / sqrtf(cta_sum(q, red + 8) / (float)W + eps);
  for (int c = threadIdx.x; c < W; c += blockDim.x) row[c] = fmaf((row[c] - mean) * inv, w[c], b[c]);
}

template <typename AT>
__global__ void __launch_bounds__(256) layernorm_add_any_kernel(const LnAdd a) {
  extern __shared__ __align__(16) float row[];   // each thread touches only its own elements of it
  __shared__ float red[4][8];
  pdl_sync();
  const int W = a.W;
  const int t = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  float* xr = a.x + (size_t)t * W;
  const float* yr = a.y ? a.y + (size_t)t * a.y_ld : nullptr;
  const bool replace = yr && !a.post_w;
  if (yr) {
    for (int c = threadIdx.x; c < W; c += blockDim.x) row[c] = yr[c];
    if (!replace) ln_shared(row, a.post_w, a.post_b, a.eps, W, red[0]);
  }
  const bool changed = yr || a.add_rows || a.add_vec;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    float v = replace ? row[c] : yr ? xr[c] + row[c] : xr[c];
    if (a.add_rows) v += a.add_rows[(size_t)t * a.add_ld + c];
    if (a.add_vec) v += a.add_vec[c];
    if (changed && !a.rows) xr[c] = v;
    row[c] = v;
  }
  if (!a.h) return;
  if (a.next_w) ln_shared(row, a.next_w, a.next_b, a.eps, W, red[2]);
  AT* hr = reinterpret_cast<AT*>(a.h) + (size_t)blockIdx.x * W;
  for (int c = threadIdx.x; c < W; c += blockDim.x) elem<AT>::store(hr + c, row[c]);
}

template <typename AT>
static cudaError_t launch_ln(const LnAdd& a, int n, cudaStream_t st) {
  const void* ptrs[] = {a.x, a.y, a.post_w, a.post_b, a.add_rows, a.add_vec, a.h, a.next_w, a.next_b};
  bool vec = a.W % 4 == 0 && a.W <= 8192 && a.y_ld % 4 == 0 && a.add_ld % 4 == 0;
  for (const void* p : ptrs) vec = vec && (reinterpret_cast<uintptr_t>(p) & 15) == 0;
  if (vec) {
    const int runs = a.W / 4, threads = runs >= 256 ? 256 : (runs + 31) / 32 * 32, nv = (runs + threads - 1) / threads;
#define PIEH_LN(NV) launch_k(layernorm_add_kernel<AT, NV>, dim3(n), dim3(threads), 0, st, a)
    return nv <= 1 ? PIEH_LN(1) : nv <= 2 ? PIEH_LN(2) : nv <= 4 ? PIEH_LN(4) : PIEH_LN(8);
#undef PIEH_LN
  }
  const size_t smem = (size_t)a.W * 4;
  if (smem > 48 * 1024) cudaFuncSetAttribute(layernorm_add_any_kernel<AT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  return launch_k(layernorm_add_any_kernel<AT>, dim3(n), dim3(256), smem, st, a);
}

}  // namespace pieh

using namespace pieh;

extern "C" int pieh_layernorm_add(float* x, const float* y, long long y_ld, const float* post_w, const float* post_b,
                                  const float* add_rows, long long add_ld, const float* add_vec, void* h, int h_dtype,
                                  const float* next_w, const float* next_b, const int32_t* rows, float eps, int n, int W,
                                  void* stream) {
  if (!x || (post_w && (!y || !post_b)) || (next_w && (!h || !next_b)) || (rows && !h)) return PIE_ENULL;
  if (n < 0 || W < 1 || (size_t)W * 4 > 200 * 1024 || y_ld < 0 || add_ld < 0) return PIE_EINVAL_SHAPE;
  if (n == 0) return PIE_OK;
  const LnAdd a{x, y, y_ld ? y_ld : W, post_w, post_b, add_rows, add_ld ? add_ld : W, add_vec, h, next_w, next_b, rows, eps, W};
  count_launch();
  cudaError_t e = cudaSuccess;
  PIEH_DISPATCH_DTYPE(h_dtype, AT, e = launch_ln<AT>(a, n, (cudaStream_t)stream));
  return status_of(e);
}
