// Causal flash-attention for prefill chunks against the paged KV cache (SURVEY §2.6 K7 "flash_prefill").
//
// The reference materialises a dense additive [T, T] mask and calls mx.fast.scaled_dot_product_attention
// on a contiguous cache (shard/server/model/llama.py:48-59, deepseek_v2.py:47-57).  Here causality is
// implicit, the cache is paged, batches are ragged (many sequences / chunks per launch) and the chunk may
// start at any context offset (chunked prefill).
//
// Tiling: CTA = 64 query rows of one (sequence, q-head), 4 warps x 16 rows; KV is walked in 64-key tiles,
// double buffered with cp.async straight from the page pool into padded (bank-conflict-free) shared memory.
// S = QK^T and O += PV run on the tensor cores through warp-level mma.m16n8k16 (bf16 in, fp32 accumulate) with
// the FA-2 register pipeline (S accumulators are re-used as the A operand of PV); softmax is online in
// registers with exp2.  NOTE: this is the legacy (HMMA) tensor path — the tcgen05/TMEM version of this
// kernel is the planned replacement; the GEMMs that dominate prefill FLOPs already run on tcgen05.
//
// SINK form (attention of sinkattn.cu for long portions): keys visible inside blocks of positions or a sliding window beside kept first
// tokens (only tiles with visible keys are walked), a bias by distance on the scores (DIST 1: slope per head, 2: table per head, in shared
// memory), a sink that joins the softmax denominator, a gate per head or element, and run-time head sizes up to DK / DV (multiples of 8; the missing key columns are zeros).  The queries are fp32: each enters the product as the sum of two bf16 numbers,
// so that the scores are those of the fp32 queries, as in the other forms.
#include "kernels.h"
#include "launch.h"
#include "ptx.cuh"
#include "sinkattn.h"

namespace b200 {

namespace {

constexpr int kBM = 64, kBN = 64, kWarps = 4, kThreads = 128;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(smem)));
}

struct SinkForm {                            // what the SINK form adds (unused otherwise)
  const float* q32;                          // [T, heads, d]
  const float* sink; const __nv_bfloat16* gate; long long ld_gate; bool gate_elem;
  const float* slopes; const float* bias; int bias_len, bias_n;      // bias_n: entries of a head's row that visible keys can reach
  int d, v, block, window, keep;
  float scale, out_mult;                     // scale multiplies the queries (scale_log2 is log2(e) alone)
};

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(smem)));
}

template <int DK, int DV, bool SINK, int DIST = 0>
__global__ void __launch_bounds__(kThreads)
flash_prefill_kernel(const __nv_bfloat16* __restrict__ q, long long q_ld_t, long long q_ld_h,
                     const __nv_bfloat16* __restrict__ kpool, const __nv_bfloat16* __restrict__ vpool,
                     const int* __restrict__ block_tables, int max_blocks, const int* __restrict__ cu_seqlens,
                     const int* __restrict__ context_lens, int num_seqs, int q_heads, int kv_heads, int page, float scale_log2,
                     __nv_bfloat16* __restrict__ out, long long o_ld_t, const SinkForm x) {
  pdl_sync();  // PDL: predecessor's writes visible; let the successor start its prologue
  constexpr int KS = DK + 8, VS = DV + 8;  // padded row strides (elements): (stride/2) % 32 == 4 -> conflict free
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [2][kBN][KS]
  __nv_bfloat16* sV = sK + 2 * kBN * KS;                               // [2][kBN][VS]
  float* sB = reinterpret_cast<float*>(sV + 2 * kBN * VS);             // [bias_n] (DIST 2)

  // ---- which (sequence, q tile) is this CTA?
  int tile = blockIdx.x, seq = 0, q0 = 0, qlen = 0;
  for (; seq < num_seqs; ++seq) {
    qlen = cu_seqlens[seq + 1] - cu_seqlens[seq];
    const int nt = (qlen + kBM - 1) / kBM;
    if (tile < nt) break;
    tile -= nt;
  }
  if (seq >= num_seqs) return;
  q0 = tile * kBM;
  const int hq = blockIdx.y;
  const int hk = hq / (q_heads / kv_heads);
  const int tok0 = cu_seqlens[seq] + q0;             // first token row of the tile
  const int rows = min(kBM, qlen - q0);
  const int ctx_after = context_lens[seq];
  const int pos0 = ctx_after - qlen + q0;            // absolute position of the tile's first query
  const int kv_end = min(ctx_after, pos0 + rows);    // causal: keys 0 .. last query position
  const int D = SINK ? x.d : DK, V = SINK ? x.v : DV;
  // SINK: key tiles that hold visible keys: those of the kept first tokens in front of the window, then from the first window key on
  auto first_key = [&](int p) {
    int lo = x.block > 0 ? p / x.block * x.block : 0;
    if (x.window > 0) lo = max(lo, p - x.window + 1);
    return lo;
  };
  const int lo0 = SINK ? first_key(pos0) : 0;
  const int nkept = SINK ? (min(x.keep, lo0) + kBN - 1) / kBN : 0, w0 = SINK ? max(nkept, lo0 / kBN) : 0;
  const int ntiles = nkept + max(0, (kv_end + kBN - 1) / kBN - w0);
  auto tile_at = [&](int i) { return SINK ? (i < nkept ? i : w0 + i - nkept) : i; };
  const int* bt = block_tables + (size_t)seq * max_blocks;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r_lo = lane >> 2, c2 = (lane & 3) * 2;

  // two threads per key row, 16-byte chunks alternating between them; the row's page is looked up one tile before its copy is issued
  const int lr = threadIdx.x >> 1, lc = threadIdx.x & 1;
  auto row_of = [&](int j) {
    const int pos = min(j * kBN + lr, kv_end - 1);         // behind the end: the last key, masked later
    return ((size_t)bt[pos / page] * kv_heads + hk) * page + (pos % page);
  };
  auto load_tile = [&](size_t row, int buf) {
    const int KC = D / 8, VC = V / 8;
    __nv_bfloat16* dK = sK + (buf * kBN + lr) * KS;
    __nv_bfloat16* dV = sV + (buf * kBN + lr) * VS;
    const __nv_bfloat16* gK = kpool + row * D;
    const __nv_bfloat16* gV = vpool + row * V;
#pragma unroll
    for (int c = 0; c < DK / 16; ++c)
      if (!SINK || 2 * c + lc < KC) cp_async16(dK + (2 * c + lc) * 8, gK + (2 * c + lc) * 8);
#pragma unroll
    for (int c = 0; c < DV / 16; ++c)
      if (!SINK || 2 * c + lc < VC) cp_async16(dV + (2 * c + lc) * 8, gV + (2 * c + lc) * 8);
    cp_async_commit();
  };

  // ---- Q fragments (A operand), straight from global memory
  uint32_t qa[DK / 16][4], ql[SINK ? DK / 16 : 1][4];          // ql: what the rounding of fp32 queries to bf16 leaves (SINK)
  {
    const int ra = warp * 16 + r_lo, rb = ra + 8;
    if constexpr (SINK) {
      const float* fa = x.q32 + ((size_t)(tok0 + ra) * q_heads + hq) * D;
      const float* fb = fa + (size_t)8 * q_heads * D;
      auto pair = [&](const float* p, bool ok, int c, uint32_t& hi, uint32_t& lo) {      // d is a multiple of 8: a pair is inside or outside as a whole
        hi = lo = 0u;
        if (!ok || c >= D) return;
        float2 f = *reinterpret_cast<const float2*>(p + c);
        f.x *= x.scale; f.y *= x.scale;
        hi = pack_bf16(f.x, f.y);
        lo = pack_bf16(f.x - __uint_as_float(hi << 16), f.y - __uint_as_float(hi & 0xffff0000u));
      };
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        pair(fa, ra < rows, ks * 16 + c2, qa[ks][0], ql[ks][0]);
        pair(fb, rb < rows, ks * 16 + c2, qa[ks][1], ql[ks][1]);
        pair(fa, ra < rows, ks * 16 + 8 + c2, qa[ks][2], ql[ks][2]);
        pair(fb, rb < rows, ks * 16 + 8 + c2, qa[ks][3], ql[ks][3]);
      }
      if (D < DK) {                            // key columns behind d: zeros in both buffers (the copies never touch them)
        const int pad = DK - D;
        for (int i = threadIdx.x; i < 2 * kBN * pad; i += kThreads) sK[(i / pad) * KS + D + i % pad] = __float2bfloat16(0.f);
      }
    } else {
    const __nv_bfloat16* qra = q + (size_t)(tok0 + ra) * q_ld_t + (size_t)hq * q_ld_h;
    const __nv_bfloat16* qrb = q + (size_t)(tok0 + rb) * q_ld_t + (size_t)hq * q_ld_h;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      qa[ks][0] = ra < rows ? *reinterpret_cast<const uint32_t*>(qra + ks * 16 + c2) : 0u;
      qa[ks][1] = rb < rows ? *reinterpret_cast<const uint32_t*>(qrb + ks * 16 + c2) : 0u;
      qa[ks][2] = ra < rows ? *reinterpret_cast<const uint32_t*>(qra + ks * 16 + 8 + c2) : 0u;
      qa[ks][3] = rb < rows ? *reinterpret_cast<const uint32_t*>(qrb + ks * 16 + 8 + c2) : 0u;
    }
    }
  }
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;
  const int qpos_a = pos0 + warp * 16 + r_lo, qpos_b = qpos_a + 8;

  const int lo_a = SINK ? first_key(qpos_a) : 0, lo_b = SINK ? first_key(qpos_b) : 0;
  load_tile(row_of(tile_at(0)), 0);
  size_t next_row = ntiles > 1 ? row_of(tile_at(1)) : 0;
  const int last_lo = SINK ? first_key(pos0 + rows - 1) : 0;
  if constexpr (DIST == 2) {                 // (the first tile's barrier comes before any use)
    for (int i = threadIdx.x; i < x.bias_n; i += kThreads) sB[i] = x.bias[(size_t)hq * x.bias_len + i];
  }
  const float slope = DIST == 1 ? x.slopes[hq] : 0.f;
  for (int j = 0; j < ntiles; ++j) {
    const int buf = j & 1;
    if (j + 1 < ntiles) {
      load_tile(next_row, buf ^ 1);
      if (j + 2 < ntiles) next_row = row_of(tile_at(j + 2));
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* tK = sK + buf * kBN * KS;
    const __nv_bfloat16* tV = sV + buf * kBN * VS;
    // ---- S = Q K^T  (16 x 64 per warp)
    float s[kBN / 8][4];
#pragma unroll
    for (int nt = 0; nt < kBN / 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
    {
      // lanes 0-7: keys nt*8 .. +7 at column ks*16, 8-15: the same keys at column +8, 16-31: the next eight keys
      const __nv_bfloat16* kr = tK + ((lane & 7) + ((lane >> 4) << 3)) * KS + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
#pragma unroll
        for (int nt = 0; nt < kBN / 8; nt += 2) {
          uint32_t kb[4];
          ldmatrix_x4(kb, kr + nt * 8 * KS + ks * 16);
          mma_bf16(s[nt], qa[ks], kb[0], kb[1]);
          mma_bf16(s[nt + 1], qa[ks], kb[2], kb[3]);
          if constexpr (SINK) {
            mma_bf16(s[nt], ql[ks], kb[0], kb[1]);
            mma_bf16(s[nt + 1], ql[ks], kb[2], kb[3]);
          }
        }
      }
    }
    // ---- mask (tiles that every row of the CTA sees as a whole need none), online softmax (base 2) on the raw scores
    const int kbase = tile_at(j) * kBN;
    if constexpr (DIST == 1) {
      const float na = (float)(kbase + c2 - qpos_a), nb = na - 8.f;          // minus the distance of the thread's first key
#pragma unroll
      for (int nt = 0; nt < kBN / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) { s[nt][e] = fmaf(slope, na + (float)(nt * 8 + e), s[nt][e]); s[nt][2 + e] = fmaf(slope, nb + (float)(nt * 8 + e), s[nt][2 + e]); }
    } else if constexpr (DIST == 2) {
      const int na = qpos_a - kbase - c2, last = x.bias_n - 1;               // keys that are not visible: any entry, masked below
#pragma unroll
      for (int nt = 0; nt < kBN / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          s[nt][e] += sB[min(max(na - nt * 8 - e, 0), last)];
          s[nt][2 + e] += sB[min(max(na + 8 - nt * 8 - e, 0), last)];
        }
    }
    float mx_a = m_a, mx_b = m_b;
    if (kbase + kBN - 1 > pos0 || (SINK && kbase < last_lo && kbase + kBN > x.keep)) {
#pragma unroll
      for (int nt = 0; nt < kBN / 8; ++nt) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int kpos = kbase + nt * 8 + c2 + e;
          if (!(kpos <= qpos_a && (!SINK || kpos >= lo_a || kpos < x.keep))) s[nt][e] = -INFINITY;
          if (!(kpos <= qpos_b && (!SINK || kpos >= lo_b || kpos < x.keep))) s[nt][2 + e] = -INFINITY;
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < kBN / 8; ++nt) {
      mx_a = fmaxf(mx_a, fmaxf(s[nt][0], s[nt][1]));
      mx_b = fmaxf(mx_b, fmaxf(s[nt][2], s[nt][3]));
    }
    mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1)); mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
    mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1)); mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
    const float ca = (mx_a == -INFINITY) ? 1.f : exp2f((m_a - mx_a) * scale_log2);
    const float cb = (mx_b == -INFINITY) ? 1.f : exp2f((m_b - mx_b) * scale_log2);
    const float ba = (mx_a == -INFINITY) ? 0.f : -mx_a * scale_log2, bb = (mx_b == -INFINITY) ? 0.f : -mx_b * scale_log2;
    float sa = 0.f, sb = 0.f;
    uint32_t pa[kBN / 16][4];
#pragma unroll
    for (int nt = 0; nt < kBN / 8; ++nt) {
      const float p0 = exp2f(fmaf(s[nt][0], scale_log2, ba)), p1 = exp2f(fmaf(s[nt][1], scale_log2, ba));
      const float p2 = exp2f(fmaf(s[nt][2], scale_log2, bb)), p3 = exp2f(fmaf(s[nt][3], scale_log2, bb));
      sa += p0 + p1; sb += p2 + p3;
      pa[nt >> 1][(nt & 1) * 2 + 0] = pack_bf16(p0, p1);
      pa[nt >> 1][(nt & 1) * 2 + 1] = pack_bf16(p2, p3);
    }
    l_a = l_a * ca + sa; l_b = l_b * cb + sb;
    m_a = mx_a; m_b = mx_b;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) { o[i][0] *= ca; o[i][1] *= ca; o[i][2] *= cb; o[i][3] *= cb; }
    // ---- O += P V
#pragma unroll
    for (int kk = 0; kk < kBN / 16; ++kk) {
#pragma unroll
      for (int nt2 = 0; nt2 < DV / 16; ++nt2) {
        uint32_t vb[4];
        // lanes 0-15: rows kk*16 + (lane & 15) at column nt2*16; lanes 16-31: same rows at column +8
        ldmatrix_x4_trans(vb, tV + (kk * 16 + (lane & 15)) * VS + nt2 * 16 + ((lane >> 4) << 3));
        mma_bf16(o[nt2 * 2], pa[kk], vb[0], vb[1]);
        mma_bf16(o[nt2 * 2 + 1], pa[kk], vb[2], vb[3]);
      }
    }
    __syncthreads();
  }
  // ---- normalise and store
  l_a += __shfl_xor_sync(0xffffffffu, l_a, 1); l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
  l_b += __shfl_xor_sync(0xffffffffu, l_b, 1); l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
  const int ra = warp * 16 + r_lo, rb = ra + 8;
  float fa = 1.f, fb = 1.f;
  if constexpr (SINK) {
    if (x.sink != nullptr) { const float sk = x.sink[hq] * 1.4426950408889634f; l_a += exp2f(fmaf(-m_a, scale_log2, sk)); l_b += exp2f(fmaf(-m_b, scale_log2, sk)); }
    fa = fb = x.out_mult;
    if (x.gate != nullptr && !x.gate_elem) {
      auto sig = [&](int r) { return 1.f / (1.f + expf(-__bfloat162float(x.gate[(size_t)(tok0 + r) * x.ld_gate + hq]))); };
      if (ra < rows) fa *= sig(ra);
      if (rb < rows) fb *= sig(rb);
    }
  }
  const float ia = l_a > 0.f ? fa / l_a : 0.f, ib = l_b > 0.f ? fb / l_b : 0.f;
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) {
    if (SINK && i * 8 >= V) break;
    if constexpr (SINK) {
      if (x.gate != nullptr && x.gate_elem) {
        const __nv_bfloat16* gp = x.gate + (size_t)(tok0 + ra) * x.ld_gate + (size_t)hq * V + i * 8 + c2;
        auto sig = [&](const __nv_bfloat16* p) { return 1.f / (1.f + expf(-__bfloat162float(*p))); };
        if (ra < rows) { o[i][0] *= sig(gp); o[i][1] *= sig(gp + 1); }
        if (rb < rows) { o[i][2] *= sig(gp + 8 * x.ld_gate); o[i][3] *= sig(gp + 8 * x.ld_gate + 1); }
      }
    }
    if (ra < rows)
      *reinterpret_cast<uint32_t*>(out + (size_t)(tok0 + ra) * o_ld_t + (size_t)hq * V + i * 8 + c2) = pack_bf16(o[i][0] * ia, o[i][1] * ia);
    if (rb < rows)
      *reinterpret_cast<uint32_t*>(out + (size_t)(tok0 + rb) * o_ld_t + (size_t)hq * V + i * 8 + c2) = pack_bf16(o[i][2] * ib, o[i][3] * ib);
  }
}

template <int DK, int DV>
cudaError_t launch_prefill(const FlashPrefillArgs& a, cudaStream_t s) {
  constexpr int smem = 2 * kBN * ((DK + 8) + (DV + 8)) * 2;
  auto kern = flash_prefill_kernel<DK, DV, false>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  dim3 grid(a.max_tiles, a.q_heads);
  (void)launch_pdl(kern, dim3(grid), dim3(kThreads), smem, s, static_cast<const __nv_bfloat16*>(a.q), a.q_ld_t, a.q_ld_h,
                                    static_cast<const __nv_bfloat16*>(a.kpool), static_cast<const __nv_bfloat16*>(a.vpool),
                                    a.block_tables, a.max_blocks, a.cu_seqlens, a.context_lens, a.num_seqs, a.q_heads, a.kv_heads,
                                    a.page, a.scale * 1.4426950408889634f, static_cast<__nv_bfloat16*>(a.out), a.o_ld_t, SinkForm{});
  return cudaGetLastError();
}

constexpr int kBiasMax = 8192;               // entries of a distance table that shared memory takes

template <int DK, int DV, int DIST>
cudaError_t launch_sink(const SinkAttnArgs& a, const int* context_lens, int max_tiles, cudaStream_t s) {
  constexpr int tiles = 2 * kBN * ((DK + 8) + (DV + 8)) * 2;
  auto kern = flash_prefill_kernel<DK, DV, true, DIST>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, tiles + (DIST == 2 ? kBiasMax * 4 : 0));
    if (e != cudaSuccess) return e;
    configured = true;
  }
  int reach = a.bias_len;                    // distances of visible keys: below the window / block unless first tokens are kept
  if (a.keep == 0 && a.window > 0 && a.window < reach) reach = a.window;
  if (a.keep == 0 && a.block > 0 && a.block < reach) reach = a.block;
  if (DIST == 2 && reach > kBiasMax) return cudaErrorInvalidValue;
  const SinkForm x{a.q, a.sink, static_cast<const __nv_bfloat16*>(a.gate), a.ld_gate, a.gate_elem, a.slopes, a.bias, a.bias_len, reach,
                   a.D, a.V, a.block, a.window, a.keep, a.scale, a.out_mult};
  kern<<<dim3(max_tiles, a.H), kThreads, tiles + (DIST == 2 ? (reach + 3) / 4 * 16 : 0), s>>>(
      nullptr, 0, 0, static_cast<const __nv_bfloat16*>(a.kpool), static_cast<const __nv_bfloat16*>(a.vpool), a.block_tables, a.max_blocks, a.cu, context_lens, a.B, a.H,
      a.G, a.page, 1.4426950408889634f, static_cast<__nv_bfloat16*>(a.out), a.ld_out, x);
  return cudaGetLastError();
}

template <int DIST>
cudaError_t launch_sink_sizes(const SinkAttnArgs& a, const int* context_lens, int max_tiles, cudaStream_t s) {
  if (a.D <= 64 && a.V <= 64) return launch_sink<64, 64, DIST>(a, context_lens, max_tiles, s);
  if (a.D <= 128) return launch_sink<128, 128, DIST>(a, context_lens, max_tiles, s);
  return launch_sink<192, 128, DIST>(a, context_lens, max_tiles, s);
}

}  // namespace

bool flash_prefill_supported(int dk, int dv) {
  return (dk == 192 && dv == 128) || (dk == 128 && dv == 128) || (dk == 64 && dv == 64);
}

cudaError_t flash_prefill_launch(const FlashPrefillArgs& a, cudaStream_t s) {
  if (a.num_seqs == 0 || a.max_tiles == 0) return cudaSuccess;
  if ((a.q_ld_t % 2) || (a.q_ld_h % 2)) return cudaErrorInvalidValue;
  if (a.dk_ == 192 && a.dv_ == 128) return launch_prefill<192, 128>(a, s);
  if (a.dk_ == 128 && a.dv_ == 128) return launch_prefill<128, 128>(a, s);
  if (a.dk_ == 64 && a.dv_ == 64) return launch_prefill<64, 64>(a, s);
  return cudaErrorNotSupported;
}

bool sink_flash_supported(int D, int V) { return D % 8 == 0 && V % 8 == 0 && D >= 8 && V >= 8 && D <= 192 && V <= 128; }
int sink_flash_bias_max() { return kBiasMax; }

cudaError_t sink_flash_launch(const SinkAttnArgs& a, const int* context_lens, int max_tiles, cudaStream_t s) {
  if (!sink_flash_supported(a.D, a.V) || a.ld_out % 2 != 0 || a.keep < 0) return cudaErrorInvalidValue;
  if (a.B == 0 || max_tiles == 0) return cudaSuccess;
  if (a.slopes != nullptr && a.bias != nullptr) return cudaErrorInvalidValue;
  if (a.slopes != nullptr) return launch_sink_sizes<1>(a, context_lens, max_tiles, s);
  if (a.bias != nullptr) return launch_sink_sizes<2>(a, context_lens, max_tiles, s);
  return launch_sink_sizes<0>(a, context_lens, max_tiles, s);
}

}  // namespace b200
