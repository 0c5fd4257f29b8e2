// Attention of single query tokens over a SHARED pool (latent attention: one cached row per position serves every head; its
// leading dv features are the value), bf16 pages.  The heads of a token are the rows of a tensor-core tile, so a cached row is
// read once for up to 16 heads instead of once per head.
//
// A CTA of 8 warps (or a cluster of 2 / 4 / 8 of them, when there are few tokens) owns one (token, group of 16 heads).  The
// visible keys -- the kept first ones the window has left behind, then the window -- are cut into slices of 16; every warp
// walks slices of its own through a private ring of cp.async stages (no CTA-wide barrier in the loop), with
//   S [16 heads x 16 keys] = Q K^T    mma.sync m16n8k16, Q and the slice through ldmatrix, rows padded by 16 bytes
//   online softmax per head in fp32 (exp2 domain), weights rounded to bf16
//   O [16 heads x dv] += P V          the same slice read transposed
// The warps' partial softmaxes meet in shared memory, the CTAs of a cluster through distributed shared memory (each CTA finishes
// some of the heads), then sink, gate and store.  Serves any key width that is a multiple of 16 and dv a multiple of 16, <= 256.
#include <cooperative_groups.h>

#include "hyb_common.cuh"
#include "hyb_mma.cuh"

namespace pieh {

namespace cg = cooperative_groups;
constexpr int kDecWarps = 8, kSlice = 16, kRows = 16;

// bytes of shared memory: Q | one ring per warp (later that warp's O) | the CTA's partial result | maxima and sums
template <int ST>
static __host__ __device__ constexpr int latent_decode_smem(int d, int dv) {
  return kRows * (2 * d + 16) + kDecWarps * ST * kSlice * (2 * d + 16) + kRows * dv * 4 + (kDecWarps + 1) * kRows * 8;
}

// DVT: dv rounded up to what the accumulators are sized for (FULL: dv is DVT); KC: d / 16 when it is fixed at compile time -- then
// the queries stay in registers --, 0: any d
template <int DVT, bool FULL, int KC, int ST, bool CLUSTER>
__global__ void __launch_bounds__(kDecWarps * 32) latent_decode_kernel(__nv_bfloat16* out, const float* q, const float* proj,
                                                                       long long ld, const pieh_bias_attn a, const pieh_batch b,
                                                                       int groups, int cs) {
  extern __shared__ __align__(16) uint8_t smem[];
  pdl_sync();
  const int d = KC ? KC * 16 : a.d, dv = FULL ? DVT : a.dv, rowb = 2 * d + 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int pair = blockIdx.x / cs, rank = blockIdx.x - pair * cs;
  const int t = pair / groups, h0 = (pair - t * groups) * kRows, nh = min(kRows, a.H - h0);
  const int i = b.tok_seq[t], p = b.tok_pos[t];
  uint8_t* ring = smem + kRows * rowb + (size_t)warp * ST * kSlice * rowb;
  float* part = reinterpret_cast<float*>(smem + kRows * rowb + kDecWarps * ST * kSlice * rowb);   // [16][dv]
  float2* wml = reinterpret_cast<float2*>(part + kRows * dv);                                      // [warps][16] (max, sum)
  float2* pml = wml + kDecWarps * kRows;                                                           // [16]
  const uint32_t sq = (uint32_t)__cvta_generic_to_shared(smem), sr = (uint32_t)__cvta_generic_to_shared(ring);

  // visible keys by number: n < kept is position n, the rest lie `gap` further on
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  const int kept = min(a.keep_first, lo), gap = lo - kept, count = p - gap + 1;
  const int slices = (count + kSlice - 1) / kSlice, per = (slices + cs - 1) / cs;
  const int s_lo = rank * per, s_hi = min(slices, s_lo + per);
  const int32_t* table = b.block_table + (size_t)i * b.bt_stride;
  const __nv_bfloat16* pool = reinterpret_cast<const __nv_bfloat16*>(a.k_pages);

  // four lanes bring a row: lane >> 2 is the row in the first half of the slice, and the one 8 further on in the second
  auto issue = [&](int sl, int st) {   // slice sl -> stage st of this warp's ring (numbers past the end repeat the last key)
    if (sl < s_hi) {
      const int na = min(sl * kSlice + (lane >> 2), count - 1), nb = min(sl * kSlice + 8 + (lane >> 2), count - 1);
      const int ja = na < kept ? na : na + gap, jb = nb < kept ? nb : nb + gap;
      const __nv_bfloat16* pa = pool + ((size_t)table[ja >> 6] * 64 + (ja & 63)) * d + (lane & 3) * 8;
      const __nv_bfloat16* pb = pool + ((size_t)table[jb >> 6] * 64 + (jb & 63)) * d + (lane & 3) * 8;
      const uint32_t da = sr + (st * kSlice + (lane >> 2)) * rowb + (lane & 3) * 16, db = da + 8 * rowb;
      if (KC > 0 && KC % 2 == 0) {
#pragma unroll
        for (int c = 0; c < KC / 2; ++c) { cp16(da + c * 64, pa + c * 32); cp16(db + c * 64, pb + c * 32); }
      } else {
        for (int c = lane & 3, k = 0; c < (d >> 3); c += 4, ++k) { cp16(da + k * 64, pa + k * 32); cp16(db + k * 64, pb + k * 32); }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int first = s_lo + warp;
#pragma unroll
  for (int k = 0; k < ST - 1; ++k) issue(first + k * kDecWarps, k);

  {   // Q: 16 threads a row, two features at a time; rows past the last head repeat it
    const int r = tid >> 4;
    const float* src = q + (size_t)t * a.q_ld + (size_t)(h0 + min(r, nh - 1)) * d;
    for (int c = 2 * (tid & 15); c < d; c += 32) *reinterpret_cast<uint32_t*>(smem + r * rowb + c * 2) = pack2(src[c], src[c + 1]);
  }
  __syncthreads();

  constexpr int OT = DVT / 8;
  constexpr float kLog2e = 1.4426950408889634f;
  const float scale2 = a.scale * kLog2e;
  float o[OT][4], m[2] = {-1e30f, -1e30f}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int x = 0; x < OT; ++x) o[x][0] = o[x][1] = o[x][2] = o[x][3] = 0.f;
  const uint32_t qa = sq + ((lane & 7) + ((lane >> 3) & 1) * 8) * rowb + (lane >> 4) * 16;
  const uint32_t k_at = ((lane & 7) + (lane >> 4) * 8) * rowb + ((lane >> 3) & 1) * 16;
  const uint32_t v_at = ((lane & 7) + ((lane >> 3) & 1) * 8) * rowb + (lane >> 4) * 16;
  uint32_t qf[KC ? KC : 1][4];
#pragma unroll
  for (int kc = 0; kc < KC; ++kc) ldsm_x4(qa + kc * 32, qf[kc][0], qf[kc][1], qf[kc][2], qf[kc][3]);
  int st = 0;
  for (int sl = first; sl < s_hi; sl += kDecWarps) {
    issue(sl + (ST - 1) * kDecWarps, st == 0 ? ST - 1 : st - 1);   // the stage that was read in the last round
    asm volatile("cp.async.wait_group %0;" ::"n"(ST - 1) : "memory");
    __syncwarp();
    const uint32_t tile = sr + st * kSlice * rowb;
    float s[2][4] = {}, u[2][4] = {};   // even and odd steps of the product: shorter dependent chains
    auto scores = [&](float (&dst)[2][4], int kc, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4(tile + k_at + kc * 32, b0, b1, b2, b3);
      mma_16816(dst[0], a0, a1, a2, a3, b0, b1);
      mma_16816(dst[1], a0, a1, a2, a3, b2, b3);
    };
    if (KC > 0) {
#pragma unroll
      for (int kc = 0; kc < KC; ++kc) scores(kc & 1 ? u : s, kc, qf[kc][0], qf[kc][1], qf[kc][2], qf[kc][3]);
    } else {
#pragma unroll 2
      for (int kc = 0; kc < (d >> 4); ++kc) {
        uint32_t a0, a1, a2, a3;
        ldsm_x4(qa + kc * 32, a0, a1, a2, a3);
        scores(s, kc, a0, a1, a2, a3);
      }
    }
    const int n0 = sl * kSlice + 2 * t4;
    float mx0 = -1e30f, mx1 = -1e30f;
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[x][e] = n0 + 8 * x + (e & 1) < count ? (s[x][e] + u[x][e]) * scale2 : -1e30f;
        if (e < 2) mx0 = fmaxf(mx0, s[x][e]); else mx1 = fmaxf(mx1, s[x][e]);
      }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1)); mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    if (mx0 > m[0] || mx1 > m[1]) {
      const float n_0 = fmaxf(m[0], mx0), n_1 = fmaxf(m[1], mx1), c0 = exp2f(m[0] - n_0), c1 = exp2f(m[1] - n_1);
      l[0] *= c0; l[1] *= c1;
#pragma unroll
      for (int x = 0; x < OT; ++x) { o[x][0] *= c0; o[x][1] *= c0; o[x][2] *= c1; o[x][3] *= c1; }
      m[0] = n_0; m[1] = n_1;
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      s[x][0] = exp2f(s[x][0] - m[0]); s[x][1] = exp2f(s[x][1] - m[0]);
      s[x][2] = exp2f(s[x][2] - m[1]); s[x][3] = exp2f(s[x][3] - m[1]);
      l[0] += s[x][0] + s[x][1]; l[1] += s[x][2] + s[x][3];
    }
    const uint32_t p0 = pack2(s[0][0], s[0][1]), p1 = pack2(s[0][2], s[0][3]), p2 = pack2(s[1][0], s[1][1]), p3 = pack2(s[1][2], s[1][3]);
#pragma unroll
    for (int x = 0; x < OT; x += 2) {
      if (FULL || x * 8 < dv) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4_trans(tile + v_at + x * 16, b0, b1, b2, b3);
        mma_16816(o[x], p0, p1, p2, p3, b0, b1);
        mma_16816(o[x + 1], p0, p1, p2, p3, b2, b3);
      }
    }
    __syncwarp();
    st = st == ST - 1 ? 0 : st + 1;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncwarp();
  // this warp's partial result over its own ring; head rows g and g + 8
  l[0] += __shfl_xor_sync(0xffffffffu, l[0], 1); l[0] += __shfl_xor_sync(0xffffffffu, l[0], 2);
  l[1] += __shfl_xor_sync(0xffffffffu, l[1], 1); l[1] += __shfl_xor_sync(0xffffffffu, l[1], 2);
  float* wo = reinterpret_cast<float*>(ring);
#pragma unroll
  for (int x = 0; x < OT; ++x) {
    const int c = x * 8 + 2 * t4;
    if (FULL || x * 8 < dv) {
      *reinterpret_cast<float2*>(wo + g * dv + c) = make_float2(o[x][0], o[x][1]);
      *reinterpret_cast<float2*>(wo + (g + 8) * dv + c) = make_float2(o[x][2], o[x][3]);
    }
  }
  if (t4 == 0) {
    wml[warp * kRows + g] = make_float2(m[0], l[0]);
    wml[warp * kRows + g + 8] = make_float2(m[1], l[1]);
  }
  __syncthreads();
  // the warps -> the CTA's partial softmax: every warp's factor first, then the sums
  if (tid < kRows) {
    float M = -1e30f, Lr = 0.f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) M = fmaxf(M, wml[w * kRows + tid].x);
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) {
      const float2 ml = wml[w * kRows + tid];
      const float f = exp2f(ml.x - M);
      Lr = fmaf(ml.y, f, Lr);
      wml[w * kRows + tid].x = f;
    }
    pml[tid] = make_float2(M, Lr);
  }
  __syncthreads();
  const int ring_f = ST * kSlice * rowb / 4;                        // floats between two warps' rings
  const float* wo0 = reinterpret_cast<const float*>(smem + kRows * rowb);
  for (int r = tid >> 4; r < nh; r += kDecWarps * 2)                // 16 threads a head, four features at a time
    for (int c = 4 * (tid & 15); c < dv; c += 64) {
      float4 A = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int w = 0; w < kDecWarps; ++w) {
        const float f = wml[w * kRows + r].x;
        const float4 v = *reinterpret_cast<const float4*>(wo0 + (size_t)w * ring_f + r * dv + c);
        A.x = fmaf(v.x, f, A.x); A.y = fmaf(v.y, f, A.y); A.z = fmaf(v.z, f, A.z); A.w = fmaf(v.w, f, A.w);
      }
      *reinterpret_cast<float4*>(part + r * dv + c) = A;
    }
  // the CTAs of the cluster (this one finishes the heads rank, rank + cs, ... of the group), the sink, the gate
  const bool has_sink = a.sinks != nullptr || a.sink != 0;
  if (CLUSTER) cg::this_cluster().sync(); else __syncthreads();
  for (int rr = tid >> 7; rank + rr * cs < nh; rr += kDecWarps / 4) {   // 128 threads a head
    const int r = rank + rr * cs, h = h0 + r;
    const float sk = (a.sinks ? a.sinks[h] : 0.f) * kLog2e;
    float f[8], M = has_sink ? sk : -1e30f, Lr = 0.f;
    if (CLUSTER) {
      cg::cluster_group cl = cg::this_cluster();
      float2 ml[8];
#pragma unroll
      for (int k = 0; k < 8; ++k)
        if (k < cs) ml[k] = cl.map_shared_rank(pml, k)[r];
#pragma unroll
      for (int k = 0; k < 8; ++k)
        if (k < cs) M = fmaxf(M, ml[k].x);
#pragma unroll
      for (int k = 0; k < 8; ++k)
        if (k < cs) { f[k] = exp2f(ml[k].x - M); Lr = fmaf(ml[k].y, f[k], Lr); }
    } else {
      M = fmaxf(M, pml[r].x);
      f[0] = exp2f(pml[r].x - M);
      Lr = pml[r].y * f[0];
    }
    if (has_sink) Lr += exp2f(sk - M);
    for (int c = tid & 127; c < dv; c += 128) {
      float A = 0.f;
      if (CLUSTER) {
        cg::cluster_group cl = cg::this_cluster();
        float v[8];
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (k < cs) v[k] = cl.map_shared_rank(part, k)[r * dv + c];
#pragma unroll
        for (int k = 0; k < 8; ++k)
          if (k < cs) A = fmaf(v[k], f[k], A);
      } else {
        A = part[r * dv + c] * f[0];
      }
      float y = A / Lr;
      if (a.g_off >= 0) y *= 1.f / (1.f + expf(-proj[(size_t)t * ld + a.g_off + (a.gate_heads ? h : (size_t)h * dv + c)]));
      out[((size_t)t * a.H + h) * dv + c] = __float2bfloat16_rn(y);
    }
  }
  if (CLUSTER) cg::this_cluster().sync();   // nobody's shared memory goes away while another CTA still reads it
}

template <int DVT, bool FULL, int KC, int ST>
static cudaError_t launch_latent_decode_t(__nv_bfloat16* out, const float* q, const float* proj, long long ld,
                                          const pieh_bias_attn& a, const pieh_batch& b, cudaStream_t st) {
  const int smem = latent_decode_smem<ST>(a.d, a.dv), groups = (a.H + kRows - 1) / kRows;
  const long long pairs = (long long)b.T * groups, want = 2LL * num_sms();
  const int cs = pairs * 8 <= want ? 8 : pairs * 4 <= want ? 4 : pairs * 2 <= want ? 2 : 1;
  auto* kern = cs == 1 ? latent_decode_kernel<DVT, FULL, KC, ST, false> : latent_decode_kernel<DVT, FULL, KC, ST, true>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(pairs * cs));
  cfg.blockDim = dim3(kDecWarps * 32);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (cs > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = cs;
    attr[n].val.clusterDim.y = attr[n].val.clusterDim.z = 1;
    ++n;
  }
  if (pdl_enabled()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  return cudaLaunchKernelEx(&cfg, kern, out, q, proj, ld, a, b, groups, cs);
}

constexpr int kDecSmemMax = 220 * 1024;

// a shared pool (the caller has checked), bf16, ordinary softmax; several heads, or there is nothing to share
bool latent_decode_ok(const pieh_bias_attn& a, const pieh_batch& b) {
  return b.T > 0 && a.d % 16 == 0 && a.dv % 16 == 0 && a.dv <= 256 && a.dv <= a.d && a.H > 1 && !a.slopes && !a.sigmoid &&
         (reinterpret_cast<uintptr_t>(a.k_pages) & 15) == 0 && latent_decode_smem<2>(a.d, a.dv) <= kDecSmemMax;
}

cudaError_t launch_latent_decode(__nv_bfloat16* out, const float* q, const float* proj, long long ld, const pieh_bias_attn& a,
                                 const pieh_batch& b, cudaStream_t st) {
  const int kc = a.d / 16;   // sizes of real models get kernels of their own
#define PIEH_LATENT(DVT, FULL, KC, ST) launch_latent_decode_t<DVT, FULL, KC, ST>(out, q, proj, ld, a, b, st)
  if (a.dv == 128 && kc == 12) return PIEH_LATENT(128, true, 12, 3);
  if (a.dv == 128 && kc == 10) return PIEH_LATENT(128, true, 10, 3);
  if (a.dv == 128 && kc == 8) return PIEH_LATENT(128, true, 8, 3);
  if (a.dv == 64 && kc == 6) return PIEH_LATENT(64, true, 6, 3);
  if (latent_decode_smem<3>(a.d, a.dv) > kDecSmemMax) return PIEH_LATENT(256, false, 0, 2);
  return a.dv <= 64 ? PIEH_LATENT(64, false, 0, 3) : a.dv <= 128 ? PIEH_LATENT(128, false, 0, 3) : PIEH_LATENT(256, false, 0, 3);
#undef PIEH_LATENT
}

}  // namespace pieh
