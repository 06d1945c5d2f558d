// Gated delta rule with ONE decay per head:  S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q  (S [N, P] per head; q, k unit
// vectors, q times q_scale; beta = sigmoid(.), g = exp(-exp(A_log) softplus(. + dt_bias))).
//
// A scalar decay commutes with everything, so tokens can be taken C at a time with the state read ONCE per C tokens: with a_i = S^T k_i and
// c_i = S^T q_i of the state S before them, G_i = g_1 .. g_i and D_mi = g_(m+1) .. g_i,
//   u_i = beta_i (v_i - G_i a_i - sum_(m<i) D_mi (k_m . k_i) u_m),   o_i = G_i c_i + sum_(m<=i) D_mi (k_m . q_i) u_m,
//   S <- G_C S + sum_m D_mC k_m u_m.
// The 2 C products with S are independent of one another, and what couples the tokens are a few numbers per head that do not depend on S:
// they come from head_delta_prepare_kernel.  (Products of decays, never quotients: a decay may underflow.)
//
// Conventions as in hybrid.cu (ragged step, state slots, a step that starts at position 0 starts from a zero state).
#include "headdelta.h"
#include "hybrid_common.cuh"

namespace b200 {
namespace {

constexpr int C = 4;                         // tokens of a group
constexpr int kCoef = 12;                    // numbers per token i and head: beta, beta G, G, D_iC | beta D_mi (k_m . k_i), m = 0 1 2 | - | D_mi (k_m . q_i), m = 0 .. 3
constexpr int kGroupsStaged = 4;             // groups per staging buffer of the scan

__device__ __forceinline__ float decay_of(float raw, float bias, float A_log) { return expf(-expf(A_log) * softplus_f(raw + bias)); }

// workspace of one group of C tokens, floats: [G][k: C, q: C][NP] (rows padded with zeros to NP) | [H][P][v: C] | [H][C][kCoef].  What a CTA of the scan
// needs of it are three runs of whole 16-byte units, whatever the sizes.
__host__ __device__ inline long long group_floats(int G, int H, int NP, int P) { return (long long)C * (2 * G * NP + H * P + H * kCoef); }
// groups of sequence b: numbers cu[b] / C + b, .. (room for the ragged ends of all sequences: T / C + B groups)
__device__ __forceinline__ int first_group(const int* cu, int b) { return cu[b] / C + b; }

// ---------------------------------------------------------------------------------------------------------- portions: token-wise operands
// One CTA per group.  A warp takes a query / key head: the products of its C keys and queries with one another, then the unit vectors.
template <typename AT, int VW>
__global__ void head_delta_prepare_kernel(HeadDeltaArgs a) {
  extern __shared__ float dots[];            // [G][6 (k_m . k_i, m < i) + 10 (k_m . q_i, m <= i)]
  const int gi = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  int lo = 0, hi = a.B - 1;
  while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (first_group(a.cu, mid) <= gi) lo = mid; else hi = mid - 1; }
  const int b = lo, s = a.cu[b], q = a.cu[b + 1] - s, j0 = (gi - first_group(a.cu, b)) * C, nt = min(C, q - j0);
  if (nt <= 0) return;
  const int N = a.N, NP = a.NP, GN = a.G * N, HP = a.H * a.P;
  const AT* in = reinterpret_cast<const AT*>(a.in) + (long long)(s + j0) * a.ld_in;
  float* ko = a.pre + (long long)gi * group_floats(a.G, a.H, NP, a.P);
  float* vo = ko + (long long)2 * C * a.G * NP;
  float* co = vo + (long long)C * HP;
  auto load = [&](const AT* p, float* f) { if constexpr (VW == 4) load4<AT>(p, f); else f[0] = ldf<AT>(p); };
  auto store = [&](float* p, const float* f) { if constexpr (VW == 4) store4<float>(p, f); else *p = f[0]; };
  for (int g = warp; g < a.G; g += nw) {
    float kk[C], qq[C], x[16];               // x: the products in the order of `dots`
#pragma unroll
    for (int i = 0; i < C; ++i) kk[i] = qq[i] = 0.f;
#pragma unroll
    for (int e = 0; e < 16; ++e) x[e] = 0.f;
    for (int n = VW * lane; n < N; n += 32 * VW) {
      float k[C][VW], w[C][VW];
#pragma unroll
      for (int i = 0; i < C; ++i) {
#pragma unroll
        for (int e = 0; e < VW; ++e) k[i][e] = w[i][e] = 0.f;
        if (i < nt) { load(in + i * a.ld_in + GN + g * N + n, k[i]); load(in + i * a.ld_in + g * N + n, w[i]); }
      }
#pragma unroll
      for (int e = 0; e < VW; ++e) {
        int z = 0;
#pragma unroll
        for (int i = 0; i < C; ++i) {
          kk[i] += k[i][e] * k[i][e]; qq[i] += w[i][e] * w[i][e];
#pragma unroll
          for (int m = 0; m < i; ++m) x[z++] += k[m][e] * k[i][e];
        }
#pragma unroll
        for (int i = 0; i < C; ++i)
#pragma unroll
          for (int m = 0; m <= i; ++m) x[z++] += k[m][e] * w[i][e];
      }
    }
    float ik[C], iq[C];
#pragma unroll
    for (int i = 0; i < C; ++i) { ik[i] = 1.f / sqrtf(warp_sum(kk[i]) + a.unit_eps); iq[i] = a.q_scale / sqrtf(warp_sum(qq[i]) + a.unit_eps); }
    int z = 0;
#pragma unroll
    for (int i = 0; i < C; ++i)
#pragma unroll
      for (int m = 0; m < i; ++m) { const float v = warp_sum(x[z]) * ik[m] * ik[i]; if (lane == 0) dots[g * 16 + z] = v; ++z; }
#pragma unroll
    for (int i = 0; i < C; ++i)
#pragma unroll
      for (int m = 0; m <= i; ++m) { const float v = warp_sum(x[z]) * ik[m] * iq[i]; if (lane == 0) dots[g * 16 + z] = v; ++z; }
    for (int n = VW * lane; n < NP; n += 32 * VW) {
#pragma unroll
      for (int i = 0; i < C; ++i) {
        float k[VW], w[VW];
#pragma unroll
        for (int e = 0; e < VW; ++e) k[e] = w[e] = 0.f;
        if (i < nt && n < N) { load(in + i * a.ld_in + GN + g * N + n, k); load(in + i * a.ld_in + g * N + n, w); }
#pragma unroll
        for (int e = 0; e < VW; ++e) { k[e] *= ik[i]; w[e] *= iq[i]; }
        store(ko + (long long)(g * 2 * C + i) * NP + n, k); store(ko + (long long)(g * 2 * C + C + i) * NP + n, w);
      }
    }
  }
  for (int e = VW * threadIdx.x; e < HP; e += VW * blockDim.x) {
    float v[C][VW];
#pragma unroll
    for (int i = 0; i < C; ++i) {
#pragma unroll
      for (int x = 0; x < VW; ++x) v[i][x] = 0.f;
      if (i < nt) load(in + i * a.ld_in + 2 * GN + e, v[i]);
    }
#pragma unroll
    for (int x = 0; x < VW; ++x) { const float f[C] = {v[0][x], v[1][x], v[2][x], v[3][x]}; store4<float>(vo + (long long)C * (e + x), f); }
  }
  __syncthreads();
  for (int h = threadIdx.x; h < a.H; h += blockDim.x) {
    const float* d = dots + (h / (a.H / a.G)) * 16;
    const float A = a.A_log[h], bias = a.dt_bias[h];
    float gd[C], bt[C];
#pragma unroll
    for (int i = 0; i < C; ++i) {
      const long long t = s + j0 + i;
      gd[i] = i < nt ? decay_of(ldf<AT>((const AT*)a.dt + t * a.ld_dt + h), bias, A) : 1.f;       // behind the end: nothing is written, nothing decays
      bt[i] = i < nt ? sigmoid_f(ldf<AT>((const AT*)a.beta + t * a.ld_b + h)) : 0.f;
    }
    float* cf = co + (long long)h * C * kCoef;
    float G = 1.f;
    int zk = 0, zq = 6;
#pragma unroll
    for (int i = 0; i < C; ++i) {
      G *= gd[i];
      float end = 1.f;
#pragma unroll
      for (int r = i + 1; r < C; ++r) end *= gd[r];
      float o[kCoef] = {bt[i], bt[i] * G, G, end, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      float D = 1.f;
#pragma unroll
      for (int lag = 0; lag <= i; ++lag) {   // D = g_(i-lag+1) .. g_i
        if (lag > 0) { D *= gd[i - lag + 1]; o[4 + i - lag] = bt[i] * D * d[zk + i - lag]; }
        o[8 + i - lag] = D * d[zq + i - lag];
      }
      zk += i; zq += i + 1;
#pragma unroll
      for (int e = 0; e < kCoef; e += 4) store4<float>(cf + i * kCoef + e, o + e);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------- portions: scan
__device__ __forceinline__ void copy_async_16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// Sums of NV values over the L lanes of a column group, halving what each lane holds: with M = min(L, NV), value v ends in the lanes l with
// l % M == v % M as d[v / M].
template <int L, int NV> __device__ __forceinline__ void fold_lanes(float (&d)[NV], int lane) {
#pragma unroll
  for (int w = 1, n = NV / 2; w < L; w <<= 1, n >>= 1) {
    if (n > 0) {
#pragma unroll
      for (int i = 0; i < n; ++i) {
        const bool odd = lane & w;
        const float keep = odd ? d[2 * i + 1] : d[2 * i], send = odd ? d[2 * i] : d[2 * i + 1];
        d[i] = keep + __shfl_xor_sync(0xffffffffu, send, w);
      }
    } else {
      d[0] += __shfl_xor_sync(0xffffffffu, d[0], w);
    }
  }
}

// State in registers: L lanes share KC value columns (a key or query fetched from shared memory serves all of them), lane l holding the key rows 4 (l + L j) + e (j < NR4, e < 4), so a warp runs 32 / L *
// KC columns.  Groups arrive by asynchronous copies into one of two buffers while the buffer before is computed; rows behind N and columns
// behind P are zeros, so the loop has no bounds checks.                       grid (B, H, ceil(P / PB)), PB = 4 * KC * 32 / L, block 128
constexpr int kScanThreads = 128;

template <int L, int NR4, int KC>
__global__ void __launch_bounds__(kScanThreads) head_delta_scan_kernel(HeadDeltaArgs a) {
  constexpr int CPW = 32 / L, NP = 4 * L * NR4, PB = kScanThreads / 32 * KC * CPW, NV = 2 * C * KC, M = L < NV ? L : NV;
  static_assert(C == 4 && (KC == 1 || KC == 2), "sums per column group: value v = token | (query << 2) | (column << 3)");
  extern __shared__ __align__(16) float smem[];
  constexpr int per = 2 * C * NP + C * PB + C * kCoef;     // floats of one group: k, q | v | coef
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l = lane % L, b = blockIdx.x, h = blockIdx.y, N = a.N, P = a.P, H = a.H, p0 = blockIdx.z * PB;
  const int g = h / (H / a.G), col = warp * KC * CPW + lane / L;          // columns col and col + CPW of the CTA's
  const int s = a.cu[b], q = a.cu[b + 1] - s;
  if (q == 0) return;
  const bool fresh = a.ctx[b] - q == 0;
  float* gS = a.state + ((long long)a.slots[b] * H + h) * N * P + p0 + col;
  bool colok[KC];
  float2 st[KC][2 * NR4];
#pragma unroll
  for (int x = 0; x < KC; ++x) {
    colok[x] = p0 + col + x * CPW < P;
#pragma unroll
    for (int j = 0; j < NR4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = 4 * (l + L * j) + e;
        const float v = (!fresh && colok[x] && n < N) ? gS[(long long)n * P + x * CPW] : 0.f;
        if (e & 1) st[x][2 * j + e / 2].y = v; else st[x][2 * j + e / 2].x = v;
      }
  }
  for (int e = threadIdx.x; e < 2 * kGroupsStaged * per; e += kScanThreads) smem[e] = 0.f;
  __syncthreads();
  const int HP = H * P, vw = min(PB, P - p0), groups = (q + C - 1) / C;
  const long long gf = group_floats(a.G, H, NP, P);
  // this thread's 16-byte units of a group: keys and queries at 4 threadIdx.x + 512 i; one unit of values or coefficients
  const float* src = a.pre + (long long)first_group(a.cu, b) * gf + 4 * threadIdx.x;
  const int extra = (int)threadIdx.x < vw ? 2 * C * a.G * NP + C * (h * P + p0) : 2 * C * a.G * NP + C * HP + h * C * kCoef - 4 * vw;
  const int xdst = 2 * C * NP + ((int)threadIdx.x < vw ? 0 : C * PB - 4 * vw) + 4 * threadIdx.x;
  const bool xok = (int)threadIdx.x < vw + C * kCoef / 4;
  src += g * 2 * C * NP;
  const float* xsrc = src - g * 2 * C * NP + extra;
  auto fetch = [&](int ng, float* buf) {     // the next ng groups
    for (int gg = 0; gg < ng; ++gg) {
      float* dst = buf + gg * per;
#pragma unroll
      for (int i = 0; i < (2 * C * NP / 4 + kScanThreads - 1) / kScanThreads; ++i)
        if (2 * C * NP / 4 % kScanThreads == 0 || 4 * (int)threadIdx.x + 4 * kScanThreads * i < 2 * C * NP)
          copy_async_16(dst + 4 * threadIdx.x + 4 * kScanThreads * i, src + 4 * kScanThreads * i);
      if (xok) copy_async_16(dst + xdst, xsrc);
      src += gf; xsrc += gf;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  static_assert(PB + C * kCoef / 4 <= kScanThreads, "one unit of values or coefficients per thread");
  fetch(min(kGroupsStaged, groups), smem);
  float* out = a.out + (long long)(s + l % C) * HP + h * P + p0 + col;       // token l % C of the group
  int left = q - l % C;                      // > 0: that token exists
  int blk = 0;
  for (int g0 = 0; g0 < groups; g0 += kGroupsStaged, ++blk) {
    const int ng = min(kGroupsStaged, groups - g0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                        // these groups have landed for every thread; the other buffer is no longer read
    if (g0 + kGroupsStaged < groups) fetch(min(kGroupsStaged, groups - g0 - kGroupsStaged), smem + ((blk + 1) & 1) * kGroupsStaged * per);
    const float* cur = smem + (blk & 1) * kGroupsStaged * per;
    for (int gg = 0; gg < ng; ++gg) {
      const float* tk = cur + gg * per;
      const float4* kq4 = reinterpret_cast<const float4*>(tk) + l;
      float2 acc[KC][2 * C];
#pragma unroll
      for (int i = 0; i < 2 * C; ++i)
#pragma unroll
        for (int x = 0; x < KC; ++x) acc[x][i] = make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < NR4; ++j)
#pragma unroll
        for (int i = 0; i < 2 * C; ++i) {
          const float4 f = kq4[i * (NP / 4) + j * L];
#pragma unroll
          for (int x = 0; x < KC; ++x) {
            acc[x][i] = fma2(st[x][2 * j], make_float2(f.x, f.y), acc[x][i]);
            acc[x][i] = fma2(st[x][2 * j + 1], make_float2(f.z, f.w), acc[x][i]);
          }
        }
      float d[NV];
#pragma unroll
      for (int v = 0; v < NV; ++v) d[v] = acc[v >> 3][v & 7].x + acc[v >> 3][v & 7].y;
      fold_lanes<L, NV>(d, lane);
      const float4* cf = reinterpret_cast<const float4*>(tk + 2 * C * NP + C * PB);
      float vt[KC][C], u[KC][C], w[KC][C], GC = 1.f;
#pragma unroll
      for (int x = 0; x < KC; ++x) {
        const float4 f = *reinterpret_cast<const float4*>(tk + 2 * C * NP + C * (col + x * CPW));
        vt[x][0] = f.x; vt[x][1] = f.y; vt[x][2] = f.z; vt[x][3] = f.w;
      }
#pragma unroll
      for (int i = 0; i < C; ++i) {
        const float4 cb = cf[3 * i], ck = cf[3 * i + 1];
#pragma unroll
        for (int x = 0; x < KC; ++x) {
          const int v = i + 8 * x;           // S^T k_i
          float t = cb.x * vt[x][i] - cb.y * __shfl_sync(0xffffffffu, d[v / M], v % M, L);
          if (i > 0) t -= ck.x * u[x][0];
          if (i > 1) t -= ck.y * u[x][1];
          if (i > 2) t -= ck.z * u[x][2];
          u[x][i] = t;
          w[x][i] = cb.w * t;
        }
        if (i == C - 1) GC = cb.z;
      }
      {                                      // the lane that holds S^T q_i finishes and stores token i
        const float G = cf[3 * (l % C)].z;
        const float4 cq = cf[3 * (l % C) + 2];
#pragma unroll
        for (int x = 0; x < NV / M; ++x) {
          const int v = x * M + l % M, c = KC == 1 ? 0 : v >> 3;      // column; lanes differ in it only when M = 16
          constexpr bool kMixed = KC == 2 && M == 16;
          const float* uc = u[kMixed ? 0 : (x * M) >> 3];
          float y = G * d[x];
          y += cq.x * (kMixed && c ? u[KC - 1][0] : uc[0]);
          y += cq.y * (kMixed && c ? u[KC - 1][1] : uc[1]);
          y += cq.z * (kMixed && c ? u[KC - 1][2] : uc[2]);
          y += cq.w * (kMixed && c ? u[KC - 1][3] : uc[3]);
          if ((v & 4) && l < NV && (c ? colok[KC - 1] : colok[0]) && left > 0) out[c * CPW] = y;
        }
        out += (long long)C * HP; left -= C;
      }
#pragma unroll
      for (int x = 0; x < KC; ++x)
#pragma unroll
        for (int j = 0; j < 2 * NR4; ++j) st[x][j] = mul2(st[x][j], make_float2(GC, GC));
#pragma unroll
      for (int j = 0; j < NR4; ++j)
#pragma unroll
        for (int i = 0; i < C; ++i) {
          const float4 f = kq4[i * (NP / 4) + j * L];
#pragma unroll
          for (int x = 0; x < KC; ++x) {
            st[x][2 * j] = fma2(make_float2(w[x][i], w[x][i]), make_float2(f.x, f.y), st[x][2 * j]);
            st[x][2 * j + 1] = fma2(make_float2(w[x][i], w[x][i]), make_float2(f.z, f.w), st[x][2 * j + 1]);
          }
        }
    }
  }
#pragma unroll
  for (int x = 0; x < KC; ++x)
#pragma unroll
    for (int j = 0; j < NR4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = 4 * (l + L * j) + e;
        if (colok[x] && n < N) gS[(long long)n * P + x * CPW] = (e & 1) ? st[x][2 * j + e / 2].y : st[x][2 * j + e / 2].x;
      }
}

// ---------------------------------------------------------------------------------------------------------- single tokens
// One token per sequence, bound by the bytes of the state: LW lanes hold VW adjacent columns each, 256 / LW rows at a time, NI times; the state
// stays in registers between the two products and the update, all its loads in flight at once.     grid (B, H, ceil(P / (LW VW))), block 256
constexpr int kStepThreads = 256;

template <typename AT, int VW, int NI>
__global__ void __launch_bounds__(kStepThreads) head_delta_step_kernel(HeadDeltaArgs a, int LW) {
  extern __shared__ float kq[];              // [N] keys | [N] queries, not yet scaled
  __shared__ float red[8][2][64], sums[8][3];
  const int b = blockIdx.x, h = blockIdx.y, N = a.N, P = a.P, H = a.H, t = a.cu[b];
  if (a.cu[b + 1] == t) return;
  const int g = h / (H / a.G), warp = threadIdx.x >> 5, lane = threadIdx.x & 31, R = kStepThreads / LW;
  const int lc = threadIdx.x % LW * VW, col = blockIdx.z * LW * VW + lc, r = threadIdx.x / LW;
  const bool fresh = a.ctx[b] == 1, colok = col < P;                 // (VW == 4: P is a multiple of 4)
  float* gS = a.state + ((long long)a.slots[b] * H + h) * N * P + col;
  float S[NI][VW];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = r + i * R;
#pragma unroll
    for (int e = 0; e < VW; ++e) S[i][e] = 0.f;
    if (!fresh && colok && n < N) {
      if constexpr (VW == 4) load4<float>(gS + (long long)n * P, S[i]); else S[i][0] = gS[(long long)n * P];
    }
  }
  const AT* row = reinterpret_cast<const AT*>(a.in) + (long long)t * a.ld_in;
  float skk = 0.f, sqq = 0.f, skq = 0.f;
  for (int n = threadIdx.x; n < N; n += kStepThreads) {
    const float kv = ldf<AT>(row + a.G * N + g * N + n), qv = ldf<AT>(row + g * N + n);
    kq[n] = kv; kq[N + n] = qv;
    skk += kv * kv; sqq += qv * qv; skq += kv * qv;
  }
  skk = warp_sum(skk); sqq = warp_sum(sqq); skq = warp_sum(skq);
  if (lane == 0) { sums[warp][0] = skk; sums[warp][1] = sqq; sums[warp][2] = skq; }
  float v[VW];
#pragma unroll
  for (int e = 0; e < VW; ++e) v[e] = colok ? ldf<AT>(row + 2 * a.G * N + h * P + col + e) : 0.f;
  const float gd = decay_of(ldf<AT>((const AT*)a.dt + (long long)t * a.ld_dt + h), a.dt_bias[h], a.A_log[h]);
  const float bt = sigmoid_f(ldf<AT>((const AT*)a.beta + (long long)t * a.ld_b + h));
  __syncthreads();
  skk = sqq = skq = 0.f;
#pragma unroll
  for (int w = 0; w < kStepThreads / 32; ++w) { skk += sums[w][0]; sqq += sums[w][1]; skq += sums[w][2]; }
  const float ik = 1.f / sqrtf(skk + a.unit_eps), iq = a.q_scale / sqrtf(sqq + a.unit_eps);
  float x[2 * VW];                           // S^T k | S^T q of this thread's columns
#pragma unroll
  for (int e = 0; e < 2 * VW; ++e) x[e] = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = min(r + i * R, N - 1);     // rows behind N hold zeros
#pragma unroll
    for (int e = 0; e < VW; ++e) { x[e] += S[i][e] * kq[n]; x[VW + e] += S[i][e] * kq[N + n]; }
  }
  for (int w = LW; w < 32; w <<= 1)
#pragma unroll
    for (int e = 0; e < 2 * VW; ++e) x[e] += __shfl_xor_sync(0xffffffffu, x[e], w);
  if (lane < LW) {
#pragma unroll
    for (int e = 0; e < VW; ++e) { red[warp][0][lc + e] = x[e]; red[warp][1][lc + e] = x[VW + e]; }
  }
  __syncthreads();
  float u[VW], y[VW];
#pragma unroll
  for (int e = 0; e < VW; ++e) {
    float ak = 0.f, aq = 0.f;
#pragma unroll
    for (int w = 0; w < kStepThreads / 32; ++w) { ak += red[w][0][lc + e]; aq += red[w][1][lc + e]; }
    u[e] = bt * (v[e] - gd * ak * ik);
    y[e] = gd * aq * iq + skq * ik * iq * u[e];
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = r + i * R;
    if (!colok || n >= N) continue;
    const float kn = kq[n] * ik;
#pragma unroll
    for (int e = 0; e < VW; ++e) S[i][e] = gd * S[i][e] + kn * u[e];
    if constexpr (VW == 4) store4<float>(gS + (long long)n * P, S[i]); else gS[(long long)n * P] = S[i][0];
  }
  if (r == 0 && colok) {
    float* o = a.out + (long long)t * H * P + h * P + col;
#pragma unroll
    for (int e = 0; e < VW; ++e) o[e] = y[e];
  }
}

template <typename K>
cudaError_t allow_smem(K k, size_t smem) {
  return smem > 48 * 1024 ? cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess;
}

int step_lanes(int P, int vw) {
  if (vw == 1) return 32;
  int lw = 4;
  while (lw < 16 && lw * 4 < P) lw *= 2;
  return lw;
}
bool step_form(const HeadDeltaArgs& a, int max_q, int& vw, int& lw) {
  vw = a.P % 4 == 0 ? 4 : 1;
  lw = step_lanes(a.P, vw);
  return max_q <= 1 && (a.N + kStepThreads / lw - 1) / (kStepThreads / lw) <= 16;
}

template <typename AT, int VW>
cudaError_t step(const HeadDeltaArgs& a, int lw, cudaStream_t s) {
  const int ni = (a.N + kStepThreads / lw - 1) / (kStepThreads / lw);
  const dim3 grid(a.B, a.H, (a.P + lw * VW - 1) / (lw * VW));
  const size_t smem = 2 * (size_t)a.N * sizeof(float);
  if (ni <= 1) head_delta_step_kernel<AT, VW, 1><<<grid, kStepThreads, smem, s>>>(a, lw);
  else if (ni <= 2) head_delta_step_kernel<AT, VW, 2><<<grid, kStepThreads, smem, s>>>(a, lw);
  else if (ni <= 4) head_delta_step_kernel<AT, VW, 4><<<grid, kStepThreads, smem, s>>>(a, lw);
  else if (ni <= 8) head_delta_step_kernel<AT, VW, 8><<<grid, kStepThreads, smem, s>>>(a, lw);
  else head_delta_step_kernel<AT, VW, 16><<<grid, kStepThreads, smem, s>>>(a, lw);
  return last();
}

template <typename AT>
cudaError_t prepare(const HeadDeltaArgs& a, cudaStream_t s) {
  const int es = (int)sizeof(AT);
  const bool vec = a.N % 4 == 0 && a.P % 4 == 0 && a.ld_in % 4 == 0 && reinterpret_cast<uintptr_t>(a.in) % (4 * es) == 0;
  const size_t smem = (size_t)a.G * 16 * sizeof(float);
  const unsigned grid = (unsigned)(a.T / C + a.B);
  cudaError_t e = vec ? allow_smem(head_delta_prepare_kernel<AT, 4>, smem) : allow_smem(head_delta_prepare_kernel<AT, 1>, smem);
  if (e != cudaSuccess) return e;
  if (vec) head_delta_prepare_kernel<AT, 4><<<grid, 256, smem, s>>>(a);
  else head_delta_prepare_kernel<AT, 1><<<grid, 256, smem, s>>>(a);
  return last();
}

// lanes per column group, steps of 4 L key rows, columns per thread and warps of the scan.  Many columns: few lanes and two columns per thread
// need the fewest instructions.  Few columns (a prompt alone): a token's time is the serial instruction count of a warp, so one column per
// thread and more lanes (not all 32: what a warp does whatever its share then weighs too much).
struct ScanShape { int L, nr4, kc; };
ScanShape scan_shape(const HeadDeltaArgs& a) {
  int L = a.N <= 64 ? 4 : a.N <= 128 ? 8 : 16, kc = 2;
  if ((long long)a.B * a.H * a.P <= 148 * 32) {
    kc = 1;
    while (L < 16 && a.N > 4 * L) L *= 2;
  }
  const int need = (a.N + 4 * L - 1) / (4 * L);
  return {L, need <= 1 ? 1 : need <= 2 ? 2 : need <= 4 ? 4 : 8, kc};
}

template <int L, int KC>
cudaError_t scan(const HeadDeltaArgs& a, const ScanShape& f, cudaStream_t s) {
  constexpr int PB = kScanThreads / 32 * KC * (32 / L);
  auto go = [&](auto k) -> cudaError_t {
    const size_t smem = 2 * (size_t)kGroupsStaged * (2 * C * a.NP + C * PB + C * kCoef) * sizeof(float);
    const cudaError_t e = allow_smem(k, smem);
    if (e != cudaSuccess) return e;
    k<<<dim3(a.B, a.H, (a.P + PB - 1) / PB), kScanThreads, smem, s>>>(a);
    return last();
  };
  if (f.nr4 == 1) return go(head_delta_scan_kernel<L, 1, KC>);
  if (f.nr4 == 2) return go(head_delta_scan_kernel<L, 2, KC>);
  if (f.nr4 == 4) return go(head_delta_scan_kernel<L, 4, KC>);
  return go(head_delta_scan_kernel<L, 8, KC>);
}

}  // namespace

bool head_delta_supported(int N) { return N >= 1 && N <= 512; }

long long head_delta_workspace(const HeadDeltaArgs& a, int max_q) {
  int vw, lw;
  if (step_form(a, max_q, vw, lw)) return 0;
  const ScanShape f = scan_shape(a);
  return (long long)(a.T / C + a.B) * group_floats(a.G, a.H, 4 * f.L * f.nr4, a.P);
}

cudaError_t head_delta_launch(HeadDeltaArgs a, bool f32, int max_q, cudaStream_t s) {
  if (a.G < 1 || a.H % a.G != 0 || a.P < 1 || !head_delta_supported(a.N) || a.G > 3000) return cudaErrorInvalidValue;
  int vw, lw;
  if (step_form(a, max_q, vw, lw)) {
    if (vw == 4) AT_DISPATCH(f32, return (step<AT, 4>(a, lw, s)));
    AT_DISPATCH(f32, return (step<AT, 1>(a, lw, s)));
  }
  if (a.pre == nullptr || (reinterpret_cast<uintptr_t>(a.pre) & 15) != 0) return cudaErrorInvalidValue;
  const ScanShape f = scan_shape(a);
  a.NP = 4 * f.L * f.nr4;
  cudaError_t e = cudaSuccess;
  AT_DISPATCH(f32, e = prepare<AT>(a, s));
  if (e != cudaSuccess) return e;
  if (f.kc == 1) return f.L == 4 ? scan<4, 1>(a, f, s) : f.L == 8 ? scan<8, 1>(a, f, s) : scan<16, 1>(a, f, s);
  return f.L == 4 ? scan<4, 2>(a, f, s) : f.L == 8 ? scan<8, 2>(a, f, s) : scan<16, 2>(a, f, s);
}
}  // namespace b200
