// Grouped-query attention over paged keys / values with a sink in the softmax: keys visible inside fixed blocks of positions or a sliding
// window, beside kept first tokens; a bias by distance (slope per head, table per head) on the scores; the result times a gate.  For steps of few query rows (decode, short portions), for exact
// mode and for any size; long bf16 portions run on the tensor cores (attention_prefill.cu).
//
// Conventions as in hybrid.cu; scores, softmax and accumulators are fp32.  The visible keys of a query at position p are numbered
// 0 .. n - 1: first the kept ones in front of its window, then the window (key_at), so loops and key splits run over visible keys only.
#include "sinkattn.h"
#include "hybrid_common.cuh"

namespace b200 {
namespace {

constexpr int kTile = 32;
constexpr float kLog2e = 1.4426950408889634f;

struct Visible {
  int lo, kept, n;                          // first key of the block / window, kept keys in front of it, number of visible keys
  __device__ __forceinline__ Visible(const SinkAttnArgs& a, int pos) {
    lo = a.block > 0 ? pos / a.block * a.block : 0;
    if (a.window > 0) lo = max(lo, pos - a.window + 1);
    kept = min(a.keep, lo);
    n = kept + pos - lo + 1;
  }
  __device__ __forceinline__ int key_at(int i) const { return i < kept ? i : lo + i - kept; }
};

// factor of element d of head h
template <typename AT> __device__ __forceinline__ float out_factor(const SinkAttnArgs& a, long long t, int h, int d) {
  return a.gate != nullptr ? a.out_mult * sigmoid_f(ldf<AT>((const AT*)a.gate + t * a.ld_gate + (a.gate_elem ? h * a.V + d : h))) : a.out_mult;
}
// added to the score of head h and a key n tokens back
__device__ __forceinline__ float distance_bias(const SinkAttnArgs& a, int h, int n) {
  float b = 0.f;
  if (a.slopes != nullptr) b -= a.slopes[h] * (float)n;
  if (a.bias != nullptr) b += a.bias[h * a.bias_len + min(n, a.bias_len - 1)];
  return b;
}

// ---------------------------------------------------------------------------------------------------------- vector form
// 2^v: the library's for exact mode, the hardware's for bf16 serving (results that the inputs' rounding drowns)
template <typename AT> __device__ __forceinline__ float exp2_of(float v);
template <> __device__ __forceinline__ float exp2_of<float>(float v) { return exp2f(v); }
template <> __device__ __forceinline__ float exp2_of<__nv_bfloat16>(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}

// 8 adjacent activations (16 bytes of bf16, 32 of float): asynchronous copy into this thread's slot of shared memory, and out of it
template <typename AT> constexpr int kChunkBytes = 8 * (int)sizeof(AT);
template <typename AT> __device__ __forceinline__ void chunk_copy(unsigned dst, const AT* src) {
#pragma unroll
  for (int i = 0; i < kChunkBytes<AT>; i += 16)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + i), "l"((const char*)src + i) : "memory");
}
__device__ __forceinline__ void chunk_get(const __nv_bfloat16* p, float2* f) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const unsigned w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) f[i] = make_float2(__uint_as_float(w[i] << 16), __uint_as_float(w[i] & 0xffff0000u));
}
__device__ __forceinline__ void chunk_get(const float* p, float2* f) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = make_float2(a.x, a.y); f[1] = make_float2(a.z, a.w); f[2] = make_float2(b.x, b.y); f[3] = make_float2(b.z, b.w);
}

constexpr int kRowWarps = 4;

// grid (tokens, G * ceil((H/G) / RG), key splits), 4 warps.  LK lanes share a key: each holds 8 adjacent entries of the key and of the value
// (dim and vdim multiples of 8, at most 8 LK), so a warp takes 32 / LK keys at a time, U of them per lane group and step, straight from the
// pages by asynchronous copies of S - 1 steps ahead — every thread reads back only what it copied itself, so no barrier is involved — and
// uses them for RG query heads.  Every lane group runs an online softmax (base 2) of its own over its keys;
// the groups are merged at the end, over the lanes of a warp by shuffles and over the warps in shared memory.  BIAS: distance_bias on the scores,
// evaluated once per key and head for the whole CTA (bias_keys > 0) or where it is used.
template <typename AT, int LK, int RG, int U, int S, bool BIAS>
__global__ void __launch_bounds__(32 * kRowWarps, RG == 4 ? 4 : 5) sink_rows_kernel(SinkAttnArgs a) {
  extern __shared__ __align__(16) unsigned char ring[];      // [S][U][key, value][thread] chunks
  constexpr int KPW = 32 / LK, STEP = kRowWarps * KPW;
  __shared__ float so[kRowWarps][RG][8 * LK];
  __shared__ float sm[kRowWarps][RG], sl[kRowWarps][RG];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, grp = lane / LK, d0 = 8 * (lane % LK);
  const int D = a.D, V = a.V, G = a.G, Rg = a.H / G, nb = (Rg + RG - 1) / RG, t = blockIdx.x;
  const int g = blockIdx.y / nb, r0 = (blockIdx.y % nb) * RG, pos = a.positions[t];
  const int* bt = a.block_tables + (long long)seq_of(a.cu, a.B, t) * a.max_blocks;
  const bool dk = d0 < D, dv = d0 < V;
  float* bias = reinterpret_cast<float*>(ring + S * U * 2 * 32 * kRowWarps * kChunkBytes<AT>);      // [bias_keys][RG], base 2
  float2 q[RG][4], o[RG][4];
  float m[RG], l[RG];
#pragma unroll
  for (int r = 0; r < RG; ++r) {
    m[r] = -INFINITY; l[r] = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) q[r][e] = o[r][e] = make_float2(0.f, 0.f);
    if (dk && r0 + r < Rg) {
      const float2* qp = reinterpret_cast<const float2*>(a.q + ((long long)t * a.H + g * Rg + r0 + r) * D + d0);
      const float f = a.scale * kLog2e;
#pragma unroll
      for (int e = 0; e < 4; ++e) q[r][e] = mul2(qp[e], make_float2(f, f));
    }
  }
  const Visible vis(a, pos);
  const long long ib = (long long)blockIdx.z * a.chunk;
  const int ibeg = (int)min(ib, (long long)vis.n), iend = (int)min((long long)vis.n, ib + a.chunk);
  const AT* kpool = (const AT*)a.kpool + d0;
  const AT* vpool = (const AT*)a.vpool + d0;
  AT* slot = reinterpret_cast<AT*>(ring) + threadIdx.x * 8;
  constexpr int kSlots = 32 * kRowWarps * 8;                  // elements between the chunks of one thread
  const unsigned slot_addr = (unsigned)__cvta_generic_to_shared(slot);
  const int first = ibeg + warp * KPW + grp, steps = max(0, (iend - (first - grp) + STEP * U - 1) / (STEP * U));      // uniform over the warp
  int pg[U], off[U];
  auto pages = [&](int k) {                   // pages of step k (behind the end: of the last key, masked later)
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int j = vis.key_at(min(first + (k * U + u) * STEP, iend - 1)), p = a.page_shift >= 0 ? j >> a.page_shift : j / a.page;
      pg[u] = bt[p];
      off[u] = j - p * a.page;
    }
  };
  auto copy = [&](int stage) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const long long row = (long long)(pg[u] * G + g) * a.page + off[u];
      const unsigned dst = slot_addr + (stage * U + u) * 2 * kSlots * (int)sizeof(AT);
      if (dk) chunk_copy<AT>(dst, kpool + row * D);
      if (dv) chunk_copy<AT>(dst + kSlots * (int)sizeof(AT), vpool + row * V);
    }
  };
  if (!dk || !dv) {                           // entries behind dim / vdim: zeros
    for (int c = 0; c < S * U; ++c)
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        if (!dk) stf<AT>(slot + 2 * c * kSlots + e, 0.f);
        if (!dv) stf<AT>(slot + (2 * c + 1) * kSlots + e, 0.f);
      }
  }
  if constexpr (BIAS) {
    if (a.bias_keys > 0) {
      for (int e = threadIdx.x; e < (iend - ibeg) * RG; e += 32 * kRowWarps) {
        const int i = e / RG, r = e % RG;
        bias[e] = r0 + r < Rg ? kLog2e * distance_bias(a, g * Rg + r0 + r, pos - vis.key_at(ibeg + i)) : 0.f;
      }
      __syncthreads();
    }
  }
  if (steps > 0) pages(0);
#pragma unroll
  for (int k = 0; k < S - 1; ++k) {
    if (k < steps) { copy(k); if (k + 1 < steps) pages(k + 1); }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  int stage = 0;
  for (int k = 0; k < steps; ++k) {
    const int i0 = first + k * U * STEP;
    asm volatile("cp.async.wait_group %0;" ::"n"(S - 2) : "memory");
    const AT* cur = slot + stage * U * 2 * kSlots;
    stage = stage + 1 == S ? 0 : stage + 1;
    float s[U * RG];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float2 f[4];
      chunk_get(cur + 2 * u * kSlots, f);
#pragma unroll
      for (int r = 0; r < RG; ++r) {
        float2 d = mul2(q[r][0], f[0]);
#pragma unroll
        for (int e = 1; e < 4; ++e) d = fma2(q[r][e], f[e], d);
        s[u * RG + r] = d.x + d.y;
      }
    }
    sum_over_lanes<U * RG, LK>(s, lane);
    if constexpr (BIAS) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = min(i0 + u * STEP, iend - 1);
        if (a.bias_keys > 0) {
          const float* b = bias + (i - ibeg) * RG;
          if constexpr (RG == 4) { const float4 f = *reinterpret_cast<const float4*>(b); s[u * RG] += f.x; s[u * RG + 1] += f.y; s[u * RG + 2] += f.z; s[u * RG + 3] += f.w; }
          else
#pragma unroll
            for (int r = 0; r < RG; ++r) s[u * RG + r] += b[r];
        } else {
          const int n = pos - vis.key_at(i);
#pragma unroll
          for (int r = 0; r < RG; ++r) if (r0 + r < Rg) s[u * RG + r] = fmaf(distance_bias(a, g * Rg + r0 + r, n), kLog2e, s[u * RG + r]);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i0 + u * STEP >= iend) {
#pragma unroll
        for (int r = 0; r < RG; ++r) s[u * RG + r] = -INFINITY;
      }
#pragma unroll
    for (int r = 0; r < RG; ++r) {
      float nm = m[r];
#pragma unroll
      for (int u = 0; u < U; ++u) nm = fmaxf(nm, s[u * RG + r]);
      const float base = nm == -INFINITY ? 0.f : nm, cf = exp2_of<AT>(m[r] - base);       // m = -inf (nothing yet): the factor is 0
      m[r] = nm;
      l[r] *= cf;
#pragma unroll
      for (int e = 0; e < 4; ++e) o[r][e] = mul2(o[r][e], make_float2(cf, cf));
#pragma unroll
      for (int u = 0; u < U; ++u) { s[u * RG + r] = exp2_of<AT>(s[u * RG + r] - base); l[r] += s[u * RG + r]; }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float2 f[4];
      chunk_get(cur + (2 * u + 1) * kSlots, f);
#pragma unroll
      for (int r = 0; r < RG; ++r)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[r][e] = fma2(make_float2(s[u * RG + r], s[u * RG + r]), f[e], o[r][e]);
    }
    // the stage read last round is free
    if (k + S - 1 < steps) { copy(stage == 0 ? S - 2 : stage == 1 ? S - 1 : stage - 2); if (k + S < steps) pages(k + S); }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  // merge the lane groups of the warp, then the warps
#pragma unroll
  for (int r = 0; r < RG; ++r) {
#pragma unroll
    for (int w = LK; w < 32; w <<= 1) {
      const float om = __shfl_xor_sync(0xffffffffu, m[r], w), ol = __shfl_xor_sync(0xffffffffu, l[r], w);
      const float nm = fmaxf(m[r], om), base = nm == -INFINITY ? 0.f : nm, c0 = exp2f(m[r] - base), c1 = exp2f(om - base);
      m[r] = nm; l[r] = l[r] * c0 + ol * c1;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        o[r][e].x = o[r][e].x * c0 + __shfl_xor_sync(0xffffffffu, o[r][e].x, w) * c1;
        o[r][e].y = o[r][e].y * c0 + __shfl_xor_sync(0xffffffffu, o[r][e].y, w) * c1;
      }
    }
    if (grp == 0) {
#pragma unroll
      for (int e = 0; e < 4; ++e) { so[warp][r][d0 + 2 * e] = o[r][e].x; so[warp][r][d0 + 2 * e + 1] = o[r][e].y; }
    }
    if (lane == 0) { sm[warp][r] = m[r]; sl[warp][r] = l[r]; }
  }
  __syncthreads();
  for (int x = threadIdx.x; x < RG * V; x += 32 * kRowWarps) {
    const int r = x / V, d = x % V, h = g * Rg + r0 + r;
    if (r0 + r >= Rg) break;
    float M = sm[0][r];
#pragma unroll
    for (int w = 1; w < kRowWarps; ++w) M = fmaxf(M, sm[w][r]);
    const float base = M == -INFINITY ? 0.f : M;
    float den = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < kRowWarps; ++w) {
      const float c = exp2f(sm[w][r] - base);
      den += sl[w][r] * c; acc += so[w][r][d] * c;
    }
    if (a.nsplit == 1) {
      if (a.sink != nullptr) den += exp2f(a.sink[h] * kLog2e - base);       // joins the denominator only: no value
      stf<AT>((AT*)a.out + (long long)t * a.ld_out + (long long)h * V + d, acc * out_factor<AT>(a, t, h, d) / den);
    } else {
      float* pp = a.part + (((long long)t * a.H + h) * a.nsplit + blockIdx.z) * (V + 2);
      pp[2 + d] = acc;
      if (d == 0) { pp[0] = M / kLog2e; pp[1] = den; }
    }
  }
}

// ---------------------------------------------------------------------------------------------------------- any size
// grid (tokens, G * ceil((H/G) / warps), key splits); one warp per query head, the warps of a CTA share one key / value head whose tile
// of kTile keys and values is staged in shared memory as floats.  Lane j scores key j of the tile; the running softmax (m, l) and the
// accumulator live in registers, lane owning the value columns lane + 32 i.
template <typename AT, int NPL>
__global__ void sink_attention_kernel(SinkAttnArgs a) {
  extern __shared__ __align__(16) float smem[];
  const int nw = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int D = a.D, V = a.V, ldk = D + 1;
  float* qs = smem;                         // [nw][D]
  float* ks = qs + nw * D;                  // [tile][D + 1]
  float* vs = ks + kTile * ldk;             // [tile][V]
  const int t = blockIdx.x, Rg = a.H / a.G, nb = (Rg + nw - 1) / nw;
  const int g = blockIdx.y / nb, r = (blockIdx.y % nb) * nw + warp, h = g * Rg + r;
  const bool valid = r < Rg;
  const int pos = a.positions[t];
  const int* bt = a.block_tables + (long long)seq_of(a.cu, a.B, t) * a.max_blocks;
  for (int i = threadIdx.x; i < nw * D; i += blockDim.x) {
    const int rr = (blockIdx.y % nb) * nw + i / D;
    qs[i] = rr < Rg ? a.q[((long long)t * a.H + g * Rg + rr) * D + i % D] * a.scale : 0.f;
  }
  float m = -INFINITY, l = 0.f, o[NPL];
#pragma unroll
  for (int i = 0; i < NPL; ++i) o[i] = 0.f;
  const float* qh = qs + warp * D;
  const Visible vis(a, pos);
  const long long ib = (long long)blockIdx.z * a.chunk;
  const int ibeg = (int)min(ib, (long long)vis.n), iend = (int)min((long long)vis.n, ib + a.chunk);
  for (int i0 = ibeg; i0 < iend; i0 += kTile) {
    __syncthreads();
    const int nk = min(kTile, iend - i0);
    for (int jj = warp; jj < nk; jj += nw) {            // each warp fetches whole rows: one block-table lookup per row
      const int j = vis.key_at(i0 + jj);
      const long long base = ((long long)bt[j / a.page] * a.G + g) * a.page + j % a.page;
      const AT* ksrc = (const AT*)a.kpool + base * D;
      const AT* vsrc = (const AT*)a.vpool + base * V;
      float* kd = ks + jj * ldk;
      float* vd = vs + jj * V;
      for (int d = lane; d < D; d += 32) kd[d] = ldf<AT>(ksrc + d);
      for (int d = lane; d < V; d += 32) vd[d] = ldf<AT>(vsrc + d);
    }
    __syncthreads();
    if (!valid) continue;
    float sc = -INFINITY;
    if (lane < nk) {
      const float* kr = ks + lane * ldk;
      float d = 0.f;
      for (int i = 0; i < D; ++i) d += qh[i] * kr[i];
      sc = d + distance_bias(a, h, pos - vis.key_at(i0 + lane));
    }
    const float nm = fmaxf(m, warp_max(sc));
    const float cf = m == -INFINITY ? 0.f : expf(m - nm);
    const float pw = lane < nk ? expf(sc - nm) : 0.f;
    l = l * cf + warp_sum(pw);
    m = nm;
#pragma unroll
    for (int i = 0; i < NPL; ++i) o[i] *= cf;
    for (int jj = 0; jj < nk; ++jj) {
      const float w = __shfl_sync(0xffffffffu, pw, jj);
      const float* vr = vs + jj * V;
#pragma unroll
      for (int i = 0; i < NPL; ++i) {
        const int d = lane + 32 * i;
        if (d < V) o[i] += w * vr[d];
      }
    }
  }
  if (!valid) return;
  if (a.nsplit == 1) {
    // the query's own position is always visible: l > 0.  The sink joins the denominator only: exp(sink - m), no value.
    if (a.sink != nullptr) l += expf(a.sink[h] - m);
    AT* orow = (AT*)a.out + (long long)t * a.ld_out + (long long)h * V;
#pragma unroll
    for (int i = 0; i < NPL; ++i) { const int d = lane + 32 * i; if (d < V) stf<AT>(orow + d, o[i] * out_factor<AT>(a, t, h, d) / l); }
  } else {
    float* pp = a.part + (((long long)t * a.H + h) * a.nsplit + blockIdx.z) * (V + 2);
    if (lane == 0) { pp[0] = m; pp[1] = l; }
#pragma unroll
    for (int i = 0; i < NPL; ++i) { const int d = lane + 32 * i; if (d < V) pp[2 + d] = o[i]; }
  }
}

// merge the key splits of one (token, head): o = sum_z o_z e^(m_z - M) / (sum_z l_z e^(m_z - M) + e^(sink - M)).  One warp each.
template <typename AT, int NPL>
__global__ void sink_combine_kernel(SinkAttnArgs a) {
  const long long th = blockIdx.x, t = th / a.H;
  const int lane = threadIdx.x, h = (int)(th % a.H), V = a.V, nsplit = a.nsplit;
  const float* pp = a.part + th * nsplit * (V + 2);
  float M = -INFINITY, den = 0.f, acc[NPL];
  for (int z = lane; z < nsplit; z += 32) M = fmaxf(M, pp[(long long)z * (V + 2)]);
  M = warp_max(M);
#pragma unroll
  for (int i = 0; i < NPL; ++i) acc[i] = 0.f;
#pragma unroll 4
  for (int z = 0; z < nsplit; ++z) {
    const float* pz = pp + (long long)z * (V + 2);
    const float e = expf(pz[0] - M);                  // a split beyond this token's keys has m = -inf: factor 0 (its o and l are 0)
    den += pz[1] * e;
#pragma unroll
    for (int i = 0; i < NPL; ++i) { const int d = lane + 32 * i; if (d < V) acc[i] += pz[2 + d] * e; }
  }
  if (a.sink != nullptr) den += expf(a.sink[h] - M);
  AT* orow = (AT*)a.out + t * a.ld_out + (long long)h * V;
#pragma unroll
  for (int i = 0; i < NPL; ++i) { const int d = lane + 32 * i; if (d < V) stf<AT>(orow + d, acc[i] * out_factor<AT>(a, t, h, d) / den); }
}

bool vector_form(int D, int V) { return D % 8 == 0 && V % 8 == 0 && D <= 256 && V <= 256; }
int heads_of(int Rg) { return Rg >= 3 ? 4 : Rg; }
int general_warps(int Rg) { return Rg < 8 ? Rg : 8; }

template <typename AT>
cudaError_t combine(const SinkAttnArgs& a, int T, cudaStream_t s) {
  const int npl = (a.V + 31) / 32;
  if (npl <= 2) sink_combine_kernel<AT, 2><<<T * a.H, 32, 0, s>>>(a);
  else if (npl <= 4) sink_combine_kernel<AT, 4><<<T * a.H, 32, 0, s>>>(a);
  else sink_combine_kernel<AT, 16><<<T * a.H, 32, 0, s>>>(a);
  return last();
}

template <typename AT, int LK, bool BIAS>
cudaError_t rows_form(const SinkAttnArgs& a, int T, cudaStream_t s) {
  const int Rg = a.H / a.G, hp = heads_of(Rg);
  const dim3 grid(T, a.G * ((Rg + hp - 1) / hp), a.nsplit);
  constexpr int U = 2, S = sizeof(AT) == 2 ? 4 : 3;
  const int smem = S * U * 2 * 32 * kRowWarps * kChunkBytes<AT> + (BIAS ? a.bias_keys * hp * (int)sizeof(float) : 0);
  auto go = [&](auto k) -> cudaError_t {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);      // static and dynamic together may pass 48 KB
    if (e != cudaSuccess) return e;
    k<<<grid, 32 * kRowWarps, smem, s>>>(a);
    return last();
  };
  if (hp == 1) return go(sink_rows_kernel<AT, LK, 1, U, S, BIAS>);
  if (hp == 2) return go(sink_rows_kernel<AT, LK, 2, U, S, BIAS>);
  return go(sink_rows_kernel<AT, LK, 4, U, S, BIAS>);
}

template <typename AT, int NPL>
cudaError_t general_form(const SinkAttnArgs& a, int T, cudaStream_t s) {
  const int nw = general_warps(a.H / a.G), nb = (a.H / a.G + nw - 1) / nw;
  const size_t smem = ((size_t)nw * a.D + (size_t)kTile * (a.D + 1) + (size_t)kTile * a.V) * sizeof(float);
  auto k = sink_attention_kernel<AT, NPL>;
  if (smem > 48 * 1024) { cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); if (e != cudaSuccess) return e; }
  k<<<dim3(T, a.G * nb, a.nsplit), 32 * nw, smem, s>>>(a);
  return last();
}

template <typename AT, bool BIAS>
cudaError_t vector_rows(const SinkAttnArgs& a, int T, cudaStream_t s) {
  const int mx = a.D > a.V ? a.D : a.V;
  return mx <= 64 ? rows_form<AT, 8, BIAS>(a, T, s) : mx <= 128 ? rows_form<AT, 16, BIAS>(a, T, s) : rows_form<AT, 32, BIAS>(a, T, s);
}

template <typename AT>
cudaError_t attention(const SinkAttnArgs& a, int T, cudaStream_t s) {
  cudaError_t e;
  const int npl = (a.V + 31) / 32;
  if (vector_form(a.D, a.V)) e = a.slopes != nullptr || a.bias != nullptr ? vector_rows<AT, true>(a, T, s) : vector_rows<AT, false>(a, T, s);
  else e = npl <= 2 ? general_form<AT, 2>(a, T, s) : npl <= 4 ? general_form<AT, 4>(a, T, s) : general_form<AT, 16>(a, T, s);
  if (e == cudaSuccess && a.nsplit > 1) e = combine<AT>(a, T, s);
  return e;
}

}  // namespace

int sink_attention_heads_per_cta(int H, int G, int D, int V) { return vector_form(D, V) ? heads_of(H / G) : general_warps(H / G); }
int sink_attention_chunk_unit() { return 32; }
int sink_attention_bias_keys() { return 2048; }

cudaError_t sink_attention_launch(const SinkAttnArgs& a, bool f32, int T, cudaStream_t s) {
  if (a.G < 1 || a.H % a.G != 0 || a.V > 512 || (size_t)(8 * a.D + kTile * (a.D + 1) + kTile * a.V) * sizeof(float) > 220 * 1024 || a.keep < 0) return cudaErrorInvalidValue;
  AT_DISPATCH(f32, return (attention<AT>(a, T, s)));
  return cudaErrorInvalidValue;
}
}  // namespace b200
