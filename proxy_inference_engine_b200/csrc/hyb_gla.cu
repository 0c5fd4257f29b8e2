// Gated linear attention over ragged steps: a matrix state S [dk, dv] per (sequence, head) in fp32, carried in a slot.
//   per token:  S <- diag(a) S + k v^T;   o = q_scale * S^T q        a in (0, 1): one decay per key channel
// gla_decay_kernel    a = sigmoid(z)^(1 / tau) with z = W2 (W1 h) + b: the narrow second product of the low-rank pair, the bias
//                     and the root in one pass, all fp32
// gla_scan_kernel     the recurrence.  A thread owns RPT state rows x CPT columns in registers (the R lanes that share a
//                     column group sit in one warp), so the token's three key-sized vectors are read from shared memory once
//                     per CPT columns; state rows are updated in pairs with the packed fp32 instructions (fma.rn.f32x2), and
//                     the read-outs of two tokens are summed over the R lanes in one exchanging butterfly (each step halves
//                     the values a lane keeps) instead of one full butterfly per value.
//                     Long portions are cut into SEGMENTS of whole 64-row tiles that run side by side: the recurrence is
//                     linear in S, so a segment acts as S_out = diag(A) S_in + B.  Pass 1 forms (A, B) per segment from a zero
//                     state, gla_carry_kernel walks every sequence's segments and leaves each one its true incoming state,
//                     pass 2 rescans the segments and writes the outputs.  Decays only ever multiply forward (every factor is
//                     at most 1), so nothing overflows whatever the decays are.
// gla_step_kernel     decoding (one row per sequence): decays, update, read-out, the head's RMS norm and the output gate in one
//                     launch; a thread-block cluster shares a head's columns and meets in distributed shared memory for the
//                     sum of squares.  The state is read and written once with 16-byte accesses.
// Everything here is fp32; only the step kernel's output is in the act dtype.
#include <cooperative_groups.h>

#include "hyb_common.cuh"

namespace pieh {

namespace cg = cooperative_groups;

// sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau).  The inner exponential only has to be good to a few ulp: its error reaches
// the result divided by tau and by 1 + e^z, and e^-z itself is the answer's order below z = -20.
__device__ __forceinline__ float root_sigmoid(float z, float inv_tau) {
  const float sp = z < -20.f ? -z : logf(1.f + __expf(-z));
  return expf(-sp * inv_tau);
}

// ---- decays ------------------------------------------------------------------------------------------------------------
constexpr int kDecayRows = 16;

// grid (ceil(C / 64 V), ceil(T / 16)): a thread keeps V neighbouring channels of 4 rows; V = 4 needs C a multiple of 4
template <int V>
__global__ void __launch_bounds__(256) gla_decay_kernel(float* decay, const float* proj, long long ld, long long low_off,
                                                        int rank, const float* w2t, const float* bias, float inv_tau, int C,
                                                        int T) {
  extern __shared__ __align__(16) float low[];   // [rank][16]
  pdl_sync();
  const int t0 = blockIdx.y * kDecayRows, nr = min(kDecayRows, T - t0);
  for (int e = threadIdx.x; e < kDecayRows * rank; e += blockDim.x) {
    const int r = e / rank, j = e - r * rank;
    low[j * kDecayRows + r] = r < nr ? proj[(size_t)(t0 + r) * ld + low_off + j] : 0.f;
  }
  const int c = (blockIdx.x * 64 + (threadIdx.x & 63)) * V, rg = (threadIdx.x >> 6) * 4;
  float z[4][V];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const float b = bias && c + v < C ? bias[c + v] : 0.f;
#pragma unroll
    for (int r = 0; r < 4; ++r) z[r][v] = b;
  }
  __syncthreads();
  if (c >= C) return;
#pragma unroll 8
  for (int j = 0; j < rank; ++j) {
    float w[V];
    if (V == 4) {
      const float4 x = *reinterpret_cast<const float4*>(w2t + (size_t)j * C + c);
      w[0] = x.x; w[1 % V] = x.y; w[2 % V] = x.z; w[3 % V] = x.w;
    } else w[0] = w2t[(size_t)j * C + c];
    const float4 l = *reinterpret_cast<const float4*>(low + j * kDecayRows + rg);
    const float lr[4] = {l.x, l.y, l.z, l.w};
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int v = 0; v < V; ++v) z[r][v] = fmaf(w[v], lr[r], z[r][v]);
  }
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    if (rg + r >= nr) break;
    float* dst = decay + (size_t)(t0 + rg + r) * C + c;
    if (V == 4)
      *reinterpret_cast<float4*>(dst) = make_float4(root_sigmoid(z[r][0], inv_tau), root_sigmoid(z[r][1 % V], inv_tau),
                                                    root_sigmoid(z[r][2 % V], inv_tau), root_sigmoid(z[r][3 % V], inv_tau));
    else dst[0] = root_sigmoid(z[r][0], inv_tau);
  }
}

// ---- the scan ----------------------------------------------------------------------------------------------------------
typedef unsigned long long f32x2;   // two fp32 in one 64-bit register
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f32x2 pair2(float lo, float hi) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void split2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }

__device__ __forceinline__ void gla_cp(float* dst, const float* src, int bytes) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  if (bytes == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

constexpr int kGlaCols = 64, kGlaChunk = 8;   // columns per CTA, tokens per shared-memory buffer

// scratch of a segmented scan: [segments, H, dk, dv] states, then [segments, H, dk] decay products.  A segment's number is
// (its first tile) / seg + (its sequence): distinct for all segments, at most (n_tiles - 1) / seg + n_seq of them.
struct GlaSeg {
  float* states;
  float* decays;
  int tiles;      // 64-row tiles per segment
};

// PASS 0: every sequence in one go (grid z = sequences).  PASS 1: a segment's (A, B).  PASS 2: a segment's outputs.
// grid (ceil(dv / 64), H, sequences | tiles)
template <int R, int RPT, int CPT, int PASS>
__global__ void __launch_bounds__(R * (kGlaCols / CPT)) gla_scan_kernel(float* o, const float* proj, long long ld,
                                                                        const float* decay, const pieh_gla d,
                                                                        const pieh_batch b, const GlaSeg sg) {
  constexpr int NT = R * (kGlaCols / CPT), DKP = R * RPT, NP = RPT / 2;
  constexpr int TOK = 3 * DKP + kGlaCols, BUF = kGlaChunk * TOK;
  static_assert(RPT % 4 == 0 && CPT % 4 == 0 && NT % 32 == 0 && R <= 32 && (R & (R - 1)) == 0, "thread tile");
  static_assert(kGlaChunk % 2 == 0, "tokens go in pairs");
  extern __shared__ __align__(16) float sm[];
  pdl_sync();
  const int h = blockIdx.y, dk = d.dk, dv = d.dv;
  int i, row0, n;
  bool from_scratch = false, to_slot = true;
  size_t seg = 0;
  if (PASS == 0) {
    i = blockIdx.z;
    row0 = b.seq_start[i];
    n = b.seq_len[i];
  } else {
    i = b.tile_seq[blockIdx.z];
    row0 = b.tile_row[blockIdx.z];
    const int start = b.seq_start[i], len = b.seq_len[i], span = 64 * sg.tiles;
    if ((row0 - start) % span) return;             // not the first tile of a segment
    const bool multi = len > span, last = row0 + span >= start + len;
    if (PASS == 1 && (!multi || last)) return;     // nothing follows: its final state comes from pass 2
    n = min(span, start + len - row0);
    seg = (size_t)(blockIdx.z / sg.tiles + i);
    from_scratch = multi;
    to_slot = last;
  }
  const int ctx = b.seq_ctx[i];
  const int rl = threadIdx.x % R, cgp = threadIdx.x / R;
  const int j0 = blockIdx.x * kGlaCols, jc = j0 + cgp * CPT;
  const size_t head = ((size_t)h * dk) * dv, whole = (size_t)d.H * dk * dv;
  float* slot = d.state + (size_t)b.seq_slot[i] * whole + head;
  float* scr = PASS == 0 ? nullptr : sg.states + seg * whole + head;

  // S2[p][c]: rows (row(p), row(p) + 1) of column jc + c; a lane's rows are RPT / 4 runs of four neighbouring ones
  f32x2 S2[NP][CPT], A2[NP];
  const float* src = PASS == 1 ? nullptr : from_scratch ? scr : (ctx > 0 ? slot : nullptr);
#pragma unroll
  for (int p = 0; p < NP; ++p) {
    const int row = (p >> 1) * 4 * R + 4 * rl + 2 * (p & 1);
    A2[p] = pair2(1.f, 1.f);
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
      const bool ok = src && jc + c < dv;
      const float lo = ok && row < dk ? src[(size_t)row * dv + jc + c] : 0.f;
      const float hi = ok && row + 1 < dk ? src[(size_t)(row + 1) * dv + jc + c] : 0.f;
      S2[p][c] = pair2(lo, hi);
    }
  }
  // rows dk .. DKP - 1 of the key-sized vectors stay zero: their state rows stay zero and add nothing
  if (DKP > dk)
    for (int e = threadIdx.x; e < 2 * kGlaChunk * 3 * (DKP - dk); e += NT) {
      const int v = e / (DKP - dk), r = e - v * (DKP - dk);
      sm[(v / 3) * TOK + (v % 3) * DKP + dk + r] = 0.f;
    }
  const bool vec = (dk & 3) == 0 && (ld & 3) == 0 && (d.k_off & 3) == 0 && (d.q_off & 3) == 0 &&
                   (reinterpret_cast<uintptr_t>(proj) & 15) == 0 && (reinterpret_cast<uintptr_t>(decay) & 15) == 0;
  const bool vvec = (dv & 3) == 0 && (ld & 3) == 0 && (d.v_off & 3) == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0;
  auto fill = [&](int which, int c0) {
    float* base = sm + which * BUF;
    const int nc = min(kGlaChunk, n - c0);
    const int step = vec ? 4 : 1, per = dk / step;
    for (int e = threadIdx.x; e < nc * per; e += NT) {
      const int tt = e / per, r = (e - tt * per) * step;
      const size_t row = (size_t)(row0 + c0 + tt);
      float* dst = base + tt * TOK + r;
      gla_cp(dst, decay + (row * d.H + h) * dk + r, 4 * step);
      gla_cp(dst + DKP, proj + row * ld + d.k_off + (size_t)h * dk + r, 4 * step);
      if (PASS != 1) gla_cp(dst + 2 * DKP, proj + row * ld + d.q_off + (size_t)h * dk + r, 4 * step);
    }
    const int vstep = vvec ? 4 : 1, vper = kGlaCols / vstep;
    for (int e = threadIdx.x; e < nc * vper; e += NT) {
      const int tt = e / vper, c = (e - tt * vper) * vstep;
      const int jj = min(j0 + c, dv - vstep);        // columns past dv hold a copy and are never stored
      gla_cp(base + tt * TOK + 3 * DKP + c, proj + (size_t)(row0 + c0 + tt) * ld + d.v_off + (size_t)h * dv + jj, 4 * vstep);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fill(0, 0);
  for (int c0 = 0, which = 0; c0 < n; c0 += kGlaChunk, which ^= 1) {
    const int nc = min(kGlaChunk, n - c0);
    if (c0 + kGlaChunk < n) {
      fill(which ^ 1, c0 + kGlaChunk);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* base = sm + which * BUF;
    auto token = [&](int tt, float* out) {
      const float* tk = base + tt * TOK;
      f32x2 a2[NP], k2[NP], q2[NP];
#pragma unroll
      for (int q = 0; q < NP / 2; ++q) {
        const int at = (q * R + rl) * 4;
        const ulonglong2 av = *reinterpret_cast<const ulonglong2*>(tk + at);
        const ulonglong2 kv = *reinterpret_cast<const ulonglong2*>(tk + DKP + at);
        a2[2 * q] = av.x; a2[2 * q + 1] = av.y;
        k2[2 * q] = kv.x; k2[2 * q + 1] = kv.y;
        if (PASS != 1) {
          const ulonglong2 qv = *reinterpret_cast<const ulonglong2*>(tk + 2 * DKP + at);
          q2[2 * q] = qv.x; q2[2 * q + 1] = qv.y;
        }
      }
      float v[CPT];
#pragma unroll
      for (int c = 0; c < CPT; c += 4) {
        const float4 x = *reinterpret_cast<const float4*>(tk + 3 * DKP + cgp * CPT + c);
        v[c] = x.x; v[c + 1] = x.y; v[c + 2] = x.z; v[c + 3] = x.w;
      }
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        const f32x2 vv = pair2(v[c], v[c]);
        f32x2 acc = 0ull;   // (0.f, 0.f)
#pragma unroll
        for (int p = 0; p < NP; ++p) {
          S2[p][c] = fma2(a2[p], S2[p][c], mul2(k2[p], vv));
          if (PASS != 1) acc = fma2(S2[p][c], q2[p], acc);
        }
        if (PASS != 1) {
          float lo, hi;
          split2(acc, lo, hi);
          out[c] = lo + hi;
        }
      }
      if (PASS == 1 && blockIdx.x == 0) {
#pragma unroll
        for (int p = 0; p < NP; ++p) A2[p] = mul2(A2[p], a2[p]);
      }
    };
#pragma unroll 1
    for (int tt = 0; tt < nc; tt += 2) {
      float val[2 * CPT];
      token(tt, val);
      if (tt + 1 < nc) token(tt + 1, val + CPT);
      else
#pragma unroll
        for (int c = 0; c < CPT; ++c) val[CPT + c] = 0.f;
      if (PASS == 1) continue;
      // exchanging butterfly over the R lanes of the column group: a lane ends with 2 CPT / R finished sums (at least one)
      int at = 0;
#pragma unroll
      for (int off = 1, m = 2 * CPT; off < R; off <<= 1) {
        if (m > 1) {
          m >>= 1;
          const bool up = rl & off;
#pragma unroll
          for (int x = 0; x < CPT; ++x) {
            if (x < m) {
              const float send = up ? val[x] : val[x + m];
              val[x] = (up ? val[x + m] : val[x]) + __shfl_xor_sync(0xffffffffu, send, off);
            }
          }
          at += up ? m : 0;
        } else {
          val[0] += __shfl_xor_sync(0xffffffffu, val[0], off);
        }
      }
      constexpr int KEEP = 2 * CPT > R ? 2 * CPT / R : 1;
      const bool writer = 2 * CPT >= R || rl < 2 * CPT;   // more lanes than sums: the upper lanes hold copies
#pragma unroll
      for (int x = 0; x < KEEP; ++x) {
        const int tok = (at + x) / CPT, col = jc + (at + x) % CPT;
        if (writer && tt + tok < nc && col < dv)
          o[((size_t)(row0 + c0 + tt + tok) * d.H + h) * dv + col] = val[x] * d.q_scale;
      }
    }
    __syncthreads();   // everyone is done with this buffer before the next fill overwrites it
  }
  float* dst = PASS == 1 ? scr : to_slot ? slot : nullptr;
  if (dst) {
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      const int row = (p >> 1) * 4 * R + 4 * rl + 2 * (p & 1);
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        if (jc + c >= dv) continue;
        float lo, hi;
        split2(S2[p][c], lo, hi);
        if (row < dk) dst[(size_t)row * dv + jc + c] = lo;
        if (row + 1 < dk) dst[(size_t)(row + 1) * dv + jc + c] = hi;
      }
    }
  }
  if (PASS == 1 && blockIdx.x == 0 && cgp == 0) {
    float* dd = sg.decays + (seg * d.H + h) * dk;
#pragma unroll
    for (int p = 0; p < NP; ++p) {
      const int row = (p >> 1) * 4 * R + 4 * rl + 2 * (p & 1);
      float lo, hi;
      split2(A2[p], lo, hi);
      if (row < dk) dd[row] = lo;
      if (row + 1 < dk) dd[row + 1] = hi;
    }
  }
}

// every segment's true incoming state, in place of its own (B) contribution; grid (ceil(H dk dv / 256), sequences)
__global__ void __launch_bounds__(256) gla_carry_kernel(const pieh_gla d, const pieh_batch b, const GlaSeg sg) {
  pdl_sync();
  const int i = blockIdx.y, len = b.seq_len[i], span = 64 * sg.tiles;
  if (len <= span) return;
  const size_t whole = (size_t)d.H * d.dk * d.dv, e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= whole) return;
  int tile = 0;
  for (int s = 0; s < i; ++s) tile += (b.seq_len[s] + 63) / 64;
  const int nseg = (len + span - 1) / span;
  const size_t row = e / d.dv, rows = (size_t)d.H * d.dk;
  float carry = b.seq_ctx[i] > 0 ? d.state[(size_t)b.seq_slot[i] * whole + e] : 0.f;
  const size_t seg = (size_t)(tile / sg.tiles + i);
  constexpr int AHEAD = 8;      // loads in flight: the chain itself is one multiply-add per segment
  for (int m0 = 0; m0 < nseg; m0 += AHEAD) {
    float own[AHEAD], a[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      own[u] = a[u] = 0.f;
      if (m0 + u + 1 < nseg) {  // nothing follows a sequence's last segment: it has no (A, B)
        own[u] = sg.states[(seg + m0 + u) * whole + e];
        a[u] = sg.decays[(seg + m0 + u) * rows + row];
      }
    }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
      if (m0 + u < nseg) {
        sg.states[(seg + m0 + u) * whole + e] = carry;
        carry = fmaf(a[u], carry, own[u]);
      }
  }
}

// ---- one row per sequence ------------------------------------------------------------------------------------------------
struct GlaStep {
  const float* w2t; const float* bias;   // decays
  long long low_off; int rank; float inv_tau;
  const float* norm_w; float eps;        // output norm and gate
  long long g_off;
};

// grid (heads x cluster, sequences); a cluster of `cs` CTAs owns one head, COLS columns each
template <typename OT, int COLS>
__global__ void __launch_bounds__(256) gla_step_kernel(OT* out, const float* proj, long long ld, const pieh_gla d,
                                                       const GlaStep g, const pieh_batch b, int cs) {
  constexpr int CG = COLS / 4, RG = 256 / CG, UN = 8;
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33], ssq;
  pdl_sync();
  const int h = blockIdx.x / cs, rank = blockIdx.x - h * cs, i = blockIdx.y;
  const int dk = d.dk, dv = d.dv, t = b.seq_start[i], ctx = b.seq_ctx[i];
  float* as = sm;              // [dk] decays
  float* ks = as + dk;         // [dk]
  float* qs = ks + dk;         // [dk]
  float* low = qs + dk;        // [rank, padded to 4]
  float* part = sm + ((3 * dk + g.rank + 3) & ~3);   // [RG][COLS]
  const int cl = threadIdx.x % CG, rg = threadIdx.x / CG;
  const int j = rank * COLS + 4 * cl;
  const bool vec = (dv & 3) == 0;
  const float* row = proj + (size_t)t * ld;
  float* S = d.state + ((size_t)b.seq_slot[i] * d.H + h) * dk * dv;
  auto load4 = [&](int r) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ctx > 0 && r < dk) {
      const float* p = S + (size_t)r * dv + j;
      if (vec) { if (j < dv) v = *reinterpret_cast<const float4*>(p); }
      else {
        if (j < dv) v.x = p[0];
        if (j + 1 < dv) v.y = p[1];
        if (j + 2 < dv) v.z = p[2];
        if (j + 3 < dv) v.w = p[3];
      }
    }
    return v;
  };
  float4 s[UN];                // the first rows of the state are on their way while the decays are formed
#pragma unroll
  for (int u = 0; u < UN; ++u) s[u] = load4(rg + u * RG);
  for (int c = threadIdx.x; c < dk; c += 256) {
    ks[c] = row[d.k_off + (size_t)h * dk + c];
    qs[c] = row[d.q_off + (size_t)h * dk + c];
  }
  for (int c = threadIdx.x; c < g.rank; c += 256) low[c] = row[g.low_off + c];
  __syncthreads();
  float v[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) v[e] = j + e < dv ? row[d.v_off + (size_t)h * dv + j + e] : 0.f;
  // decay logits: `cuts` threads share a channel's low-rank sum where the head is narrower than the CTA
  const int cuts = dk <= 64 ? 4 : dk <= 128 ? 2 : 1, span = 256 / cuts;
  const size_t C = (size_t)d.H * dk;
  for (int c = threadIdx.x % span; c < dk; c += span) {
    const size_t ch = (size_t)h * dk + c;
    float z = 0.f;
#pragma unroll 16
    for (int r = threadIdx.x / span; r < g.rank; r += cuts) z = fmaf(g.w2t[r * C + ch], low[r], z);
    part[(threadIdx.x / span) * dk + c] = z;       // cuts * dk <= 512 floats
  }
  __syncthreads();
  for (int c = threadIdx.x; c < dk; c += 256) {
    float z = g.bias ? g.bias[(size_t)h * dk + c] : 0.f;
    for (int k = 0; k < cuts; ++k) z += part[k * dk + c];
    as[c] = root_sigmoid(z, g.inv_tau);
  }
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int r0 = rg; r0 < dk; r0 += UN * RG) {
    if (r0 != rg) {
#pragma unroll
      for (int u = 0; u < UN; ++u) s[u] = load4(r0 + u * RG);
    }
#pragma unroll
    for (int u = 0; u < UN; ++u) {
      const int r = r0 + u * RG;
      if (r < dk) {
        const float a = as[r], k = ks[r], q = qs[r];
        s[u].x = fmaf(a, s[u].x, k * v[0]); s[u].y = fmaf(a, s[u].y, k * v[1]);
        s[u].z = fmaf(a, s[u].z, k * v[2]); s[u].w = fmaf(a, s[u].w, k * v[3]);
        acc.x = fmaf(s[u].x, q, acc.x); acc.y = fmaf(s[u].y, q, acc.y);
        acc.z = fmaf(s[u].z, q, acc.z); acc.w = fmaf(s[u].w, q, acc.w);
        float* p = S + (size_t)r * dv + j;
        if (vec) { if (j < dv) *reinterpret_cast<float4*>(p) = s[u]; }
        else {
          if (j < dv) p[0] = s[u].x;
          if (j + 1 < dv) p[1] = s[u].y;
          if (j + 2 < dv) p[2] = s[u].z;
          if (j + 3 < dv) p[3] = s[u].w;
        }
      }
    }
  }
  *reinterpret_cast<float4*>(part + rg * COLS + 4 * cl) = acc;
  __syncthreads();
  float oc = 0.f;
  const int col = rank * COLS + threadIdx.x;
  if (threadIdx.x < COLS) {
#pragma unroll 8
    for (int r = 0; r < RG; ++r) oc += part[r * COLS + threadIdx.x];
    oc = col < dv ? oc * d.q_scale : 0.f;
  }
  const float mine = block_sum(oc * oc, red);
  float total = mine;
  if (cs > 1) {
    cg::cluster_group cl_g = cg::this_cluster();
    if (threadIdx.x == 0) ssq = mine;
    cl_g.sync();
    total = 0.f;
    for (int r = 0; r < cs; ++r) total += *cl_g.map_shared_rank(&ssq, r);
  }
  if (threadIdx.x < COLS && col < dv) {
    const float inv = 1.f / sqrtf(total / (float)dv + g.eps);
    elem<OT>::store(out + ((size_t)t * d.H + h) * dv + col,
                    oc * inv * g.norm_w[col] * silu_f(row[g.g_off + (size_t)h * dv + col]));
  }
  if (cs > 1) cg::this_cluster().sync();   // nobody's shared memory goes away while another CTA still reads it
}

static bool gla_ok(const pieh_gla* d) {
  return d && d->H > 0 && d->H <= 65535 && d->dk > 0 && d->dk <= 512 && d->dv > 0 && d->dv <= 65535 && d->q_off >= 0 &&
         d->k_off >= 0 && d->v_off >= 0 && d->state;
}

template <int R, int RPT, int CPT, int PASS>
static cudaError_t launch_gla(float* o, const float* proj, long long ld, const float* decay, const pieh_gla& d,
                              const pieh_batch& b, const GlaSeg& sg, cudaStream_t st) {
  constexpr int NT = R * (kGlaCols / CPT);
  constexpr size_t smem = (size_t)2 * kGlaChunk * (3 * R * RPT + kGlaCols) * 4;
  static unsigned long long configured = 0;
  int dev = 0;
  cudaGetDevice(&dev);
  if (smem > 48 * 1024 && !(configured >> (dev & 63) & 1)) {
    cudaError_t e = cudaFuncSetAttribute(gla_scan_kernel<R, RPT, CPT, PASS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    configured |= 1ull << (dev & 63);
  }
  count_launch();
  return launch_k(gla_scan_kernel<R, RPT, CPT, PASS>, dim3((d.dv + kGlaCols - 1) / kGlaCols, d.H, PASS == 0 ? b.n_seq : b.n_tiles),
                  dim3(NT), smem, st, o, proj, ld, decay, d, b, sg);
}

template <int PASS>
static cudaError_t launch_gla_size(float* o, const float* proj, long long ld, const float* decay, const pieh_gla& d,
                                   const pieh_batch& b, const GlaSeg& sg, cudaStream_t st) {
  if (d.dk <= 32) return launch_gla<4, 8, 8, PASS>(o, proj, ld, decay, d, b, sg, st);
  if (d.dk <= 64) return launch_gla<8, 8, 8, PASS>(o, proj, ld, decay, d, b, sg, st);
  if (d.dk <= 128) return launch_gla<16, 8, 8, PASS>(o, proj, ld, decay, d, b, sg, st);
  if (d.dk <= 256) return launch_gla<32, 8, 8, PASS>(o, proj, ld, decay, d, b, sg, st);
  return launch_gla<32, 16, 4, PASS>(o, proj, ld, decay, d, b, sg, st);
}

}  // namespace pieh

using namespace pieh;

extern "C" int pieh_gla_decay(float* decay, const float* proj, long long ld, long long low_off, int rank, const float* w2t,
                              const float* bias, float inv_tau, int C, int T, void* stream) {
  if (!decay || !proj || !w2t) return PIE_ENULL;
  if (T < 0 || C < 1 || rank < 1 || rank > 1024 || low_off < 0 || !(inv_tau > 0.f)) return PIE_EINVAL_SHAPE;
  if (T == 0) return PIE_OK;
  const size_t smem = (size_t)kDecayRows * rank * 4;   // at most 64 KB
  const bool vec = C % 4 == 0 && ((reinterpret_cast<uintptr_t>(decay) | reinterpret_cast<uintptr_t>(w2t)) & 15) == 0;
  auto kernel = vec ? gla_decay_kernel<4> : gla_decay_kernel<1>;
  const int per = vec ? 256 : 64;
  cudaError_t e = cudaSuccess;
  if (smem > 48 * 1024) e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return status_of(e);
  count_launch();
  return status_of(launch_k(kernel, dim3((C + per - 1) / per, (T + kDecayRows - 1) / kDecayRows), dim3(256), smem,
                            (cudaStream_t)stream, decay, proj, ld, low_off, rank, w2t, bias, inv_tau, C, T));
}

extern "C" int pieh_gla_scan(float* o, const float* proj, long long ld, const float* decay, const pieh_gla* d,
                             const pieh_batch* b, float* scratch, int seg_tiles, void* stream) {
  if (!o || !proj || !decay || !d || !b) return PIE_ENULL;
  if (!gla_ok(d) || b->n_seq > 65535) return PIE_EINVAL_SHAPE;
  if (b->T == 0) return PIE_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const bool cut = scratch && seg_tiles > 0 && b->n_tiles > b->n_seq && b->tile_seq && b->tile_row && b->n_tiles <= 65535;
  GlaSeg sg = {};
  if (!cut) return status_of(launch_gla_size<0>(o, proj, ld, decay, *d, *b, sg, st));
  const size_t whole = (size_t)d->H * d->dk * d->dv, ns = (size_t)((b->n_tiles - 1) / seg_tiles + b->n_seq);
  sg.states = scratch;
  sg.decays = scratch + ns * whole;
  sg.tiles = seg_tiles;
  cudaError_t e = launch_gla_size<1>(o, proj, ld, decay, *d, *b, sg, st);
  if (e == cudaSuccess) {
    count_launch();
    e = launch_k(gla_carry_kernel, dim3((unsigned)((whole + 255) / 256), b->n_seq), dim3(256), 0, st, *d, *b, sg);
  }
  if (e == cudaSuccess) e = launch_gla_size<2>(o, proj, ld, decay, *d, *b, sg, st);
  return status_of(e);
}

extern "C" int pieh_gla_step(void* out, int out_dtype, const float* proj, long long ld, long long low_off, int rank,
                             const float* w2t, const float* bias, float inv_tau, long long g_off, const float* norm_w,
                             float eps, const pieh_gla* d, const pieh_batch* b, void* stream) {
  if (!out || !proj || !w2t || !norm_w || !d || !b) return PIE_ENULL;
  if (!gla_ok(d) || d->dv > 1024 || rank < 1 || rank > 1024 || low_off < 0 || g_off < 0 || !(inv_tau > 0.f) ||
      b->n_seq > 65535 || b->T != b->n_seq)
    return PIE_EINVAL_SHAPE;
  if (b->T == 0) return PIE_OK;
  const GlaStep g{w2t, bias, low_off, rank, inv_tau, norm_w, eps, g_off};
  // columns per CTA: 32 where that still leaves a cluster of at most 8 and the GPU is not full with 64, 128 for wide heads
  int cols = d->dv > 512 ? 128 : 64;
  if (d->dv <= 256 && (long long)b->n_seq * d->H * ((d->dv + 63) / 64) < num_sms()) cols = 32;
  int cs = 1;
  while (cs * cols < d->dv) cs <<= 1;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(d->H * cs), b->n_seq);
  cfg.blockDim = dim3(256);
  cfg.dynamicSmemBytes = (size_t)(((3 * d->dk + rank + 3) & ~3) + 1024) * 4;   // the partial read-outs: RG x COLS = 1024 floats
  cfg.stream = (cudaStream_t)stream;
  cudaLaunchAttribute attr[2];
  int na = 0;
  if (cs > 1) {
    attr[na].id = cudaLaunchAttributeClusterDimension;
    attr[na].val.clusterDim.x = cs;
    attr[na].val.clusterDim.y = 1;
    attr[na].val.clusterDim.z = 1;
    ++na;
  }
  if (pdl_enabled()) {
    attr[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  cfg.attrs = attr;
  cfg.numAttrs = na;
  count_launch();
  cudaError_t e = cudaSuccess;
  PIEH_DISPATCH_DTYPE(out_dtype, OT, {
    e = cols == 32 ? cudaLaunchKernelEx(&cfg, gla_step_kernel<OT, 32>, (OT*)out, proj, ld, *d, g, *b, cs)
        : cols == 64 ? cudaLaunchKernelEx(&cfg, gla_step_kernel<OT, 64>, (OT*)out, proj, ld, *d, g, *b, cs)
                     : cudaLaunchKernelEx(&cfg, gla_step_kernel<OT, 128>, (OT*)out, proj, ld, *d, g, *b, cs);
  });
  return status_of(e);
}
