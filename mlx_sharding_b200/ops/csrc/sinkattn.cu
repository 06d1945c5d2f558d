// Grouped-query attention over paged keys / values with a sink in the softmax: keys visible inside fixed blocks of positions or a sliding
// window, beside kept first tokens; the result of a head times a gate.  For steps of few query rows (decode, short portions), for exact
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

template <typename AT> __device__ __forceinline__ float head_factor(const SinkAttnArgs& a, long long t, int h) {
  return a.gate != nullptr ? a.out_mult * sigmoid_f(ldf<AT>((const AT*)a.gate + t * a.ld_gate + h)) : a.out_mult;
}

// ---------------------------------------------------------------------------------------------------------- vector form
// E activations (16 bytes of bf16, 32 of float) as raw registers
template <typename AT> struct Chunk8;
template <> struct Chunk8<__nv_bfloat16> {
  uint4 a;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { a = __ldg(reinterpret_cast<const uint4*>(p)); }
  __device__ __forceinline__ void zero() { a = make_uint4(0u, 0u, 0u, 0u); }
  __device__ __forceinline__ void get(float* f) const { unpack16<__nv_bfloat16>(a, f); }
};
template <> struct Chunk8<float> {
  uint4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = __ldg(reinterpret_cast<const uint4*>(p)); b = __ldg(reinterpret_cast<const uint4*>(p) + 1);
  }
  __device__ __forceinline__ void zero() { a = b = make_uint4(0u, 0u, 0u, 0u); }
  __device__ __forceinline__ void get(float* f) const { unpack16<float>(a, f); unpack16<float>(b, f + 4); }
};

constexpr int kRowWarps = 4;

// grid (tokens, G * ceil((H/G) / RG), key splits), 4 warps.  LK lanes share a key: each holds 8 adjacent entries of the key and of the value
// (dim and vdim multiples of 8, at most 8 LK), so a warp reads 32 / LK keys at a time straight from the pages with 16-byte loads, U of them
// per lane group in flight, and uses them for RG query heads.  Every lane group runs an online softmax (base 2) of its own over its keys;
// the groups are merged at the end, over the lanes of a warp by shuffles and over the warps in shared memory.
template <typename AT, int LK, int RG, int U>
__global__ void __launch_bounds__(32 * kRowWarps) sink_rows_kernel(SinkAttnArgs a) {
  constexpr int KPW = 32 / LK, STEP = kRowWarps * KPW;
  __shared__ float so[kRowWarps][RG][8 * LK];
  __shared__ float sm[kRowWarps][RG], sl[kRowWarps][RG];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, grp = lane / LK, d0 = 8 * (lane % LK);
  const int D = a.D, V = a.V, G = a.G, Rg = a.H / G, nb = (Rg + RG - 1) / RG, t = blockIdx.x;
  const int g = blockIdx.y / nb, r0 = (blockIdx.y % nb) * RG, pos = a.positions[t];
  const int* bt = a.block_tables + (long long)seq_of(a.cu, a.B, t) * a.max_blocks;
  const bool dk = d0 < D, dv = d0 < V;
  float q[RG][8], o[RG][8], m[RG], l[RG];
#pragma unroll
  for (int r = 0; r < RG; ++r) {
    m[r] = -INFINITY; l[r] = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) { q[r][e] = 0.f; o[r][e] = 0.f; }
    if (dk && r0 + r < Rg) {
      const float4* qp = reinterpret_cast<const float4*>(a.q + ((long long)t * a.H + g * Rg + r0 + r) * D + d0);
      const float4 x = qp[0], y = qp[1];
      const float f = a.scale * kLog2e;
      q[r][0] = x.x * f; q[r][1] = x.y * f; q[r][2] = x.z * f; q[r][3] = x.w * f;
      q[r][4] = y.x * f; q[r][5] = y.y * f; q[r][6] = y.z * f; q[r][7] = y.w * f;
    }
  }
  const Visible vis(a, pos);
  const long long ib = (long long)blockIdx.z * a.chunk;
  const int ibeg = (int)min(ib, (long long)vis.n), iend = (int)min((long long)vis.n, ib + a.chunk);
  const AT* kpool = (const AT*)a.kpool;
  const AT* vpool = (const AT*)a.vpool;
  for (int i0 = ibeg + warp * KPW + grp; i0 - grp < iend; i0 += STEP * U) {       // the bound is uniform over the warp
    Chunk8<AT> kc[U], vc[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * STEP, j = vis.key_at(min(i, iend - 1));
      const long long row = ((long long)bt[j / a.page] * G + g) * a.page + j % a.page;
      if (dk) kc[u].load(kpool + row * D + d0); else kc[u].zero();
      if (dv) vc[u].load(vpool + row * V + d0); else vc[u].zero();
    }
    float s[U][RG];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float f[8];
      kc[u].get(f);
#pragma unroll
      for (int r = 0; r < RG; ++r) {
        float d = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) d += q[r][e] * f[e];
        s[u][r] = d;
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int r = 0; r < RG; ++r) {
#pragma unroll
        for (int w = LK / 2; w > 0; w >>= 1) s[u][r] += __shfl_xor_sync(0xffffffffu, s[u][r], w);
        if (i0 + u * STEP >= iend) s[u][r] = -INFINITY;
      }
#pragma unroll
    for (int r = 0; r < RG; ++r) {
      float nm = m[r];
#pragma unroll
      for (int u = 0; u < U; ++u) nm = fmaxf(nm, s[u][r]);
      const float base = nm == -INFINITY ? 0.f : nm, cf = exp2f(m[r] - base);       // m = -inf (nothing yet): the factor is 0
      m[r] = nm;
      l[r] *= cf;
#pragma unroll
      for (int e = 0; e < 8; ++e) o[r][e] *= cf;
#pragma unroll
      for (int u = 0; u < U; ++u) { s[u][r] = exp2f(s[u][r] - base); l[r] += s[u][r]; }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float f[8];
      vc[u].get(f);
#pragma unroll
      for (int r = 0; r < RG; ++r)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[r][e] += s[u][r] * f[e];
    }
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
      for (int e = 0; e < 8; ++e) o[r][e] = o[r][e] * c0 + __shfl_xor_sync(0xffffffffu, o[r][e], w) * c1;
    }
    if (grp == 0) {
#pragma unroll
      for (int e = 0; e < 8; ++e) so[warp][r][d0 + e] = o[r][e];
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
      stf<AT>((AT*)a.out + (long long)t * a.ld_out + (long long)h * V + d, acc * head_factor<AT>(a, t, h) / den);
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
      sc = d;
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
    const float f = head_factor<AT>(a, t, h) / l;
    AT* orow = (AT*)a.out + (long long)t * a.ld_out + (long long)h * V;
#pragma unroll
    for (int i = 0; i < NPL; ++i) { const int d = lane + 32 * i; if (d < V) stf<AT>(orow + d, o[i] * f); }
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
  const float f = head_factor<AT>(a, t, h) / den;
  AT* orow = (AT*)a.out + t * a.ld_out + (long long)h * V;
#pragma unroll
  for (int i = 0; i < NPL; ++i) { const int d = lane + 32 * i; if (d < V) stf<AT>(orow + d, acc[i] * f); }
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

template <typename AT, int LK>
cudaError_t rows_form(const SinkAttnArgs& a, int T, cudaStream_t s) {
  const int Rg = a.H / a.G, hp = heads_of(Rg);
  const dim3 grid(T, a.G * ((Rg + hp - 1) / hp), a.nsplit);
  constexpr int U = sizeof(AT) == 2 ? 4 : 2;
  if (hp == 1) sink_rows_kernel<AT, LK, 1, U><<<grid, 32 * kRowWarps, 0, s>>>(a);
  else if (hp == 2) sink_rows_kernel<AT, LK, 2, U><<<grid, 32 * kRowWarps, 0, s>>>(a);
  else sink_rows_kernel<AT, LK, 4, U><<<grid, 32 * kRowWarps, 0, s>>>(a);
  return last();
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

template <typename AT>
cudaError_t attention(const SinkAttnArgs& a, int T, cudaStream_t s) {
  cudaError_t e;
  const int mx = a.D > a.V ? a.D : a.V, npl = (a.V + 31) / 32;
  if (vector_form(a.D, a.V)) e = mx <= 64 ? rows_form<AT, 8>(a, T, s) : mx <= 128 ? rows_form<AT, 16>(a, T, s) : rows_form<AT, 32>(a, T, s);
  else e = npl <= 2 ? general_form<AT, 2>(a, T, s) : npl <= 4 ? general_form<AT, 4>(a, T, s) : general_form<AT, 16>(a, T, s);
  if (e == cudaSuccess && a.nsplit > 1) e = combine<AT>(a, T, s);
  return e;
}

}  // namespace

int sink_attention_heads_per_cta(int H, int G, int D, int V) { return vector_form(D, V) ? heads_of(H / G) : general_warps(H / G); }
int sink_attention_chunk_unit() { return 32; }

cudaError_t sink_attention_launch(const SinkAttnArgs& a, bool f32, int T, cudaStream_t s) {
  if (a.G < 1 || a.H % a.G != 0 || a.V > 512 || (size_t)(8 * a.D + kTile * (a.D + 1) + kTile * a.V) * sizeof(float) > 220 * 1024 || a.keep < 0) return cudaErrorInvalidValue;
  AT_DISPATCH(f32, return (attention<AT>(a, T, s)));
  return cudaErrorInvalidValue;
}
}  // namespace b200
