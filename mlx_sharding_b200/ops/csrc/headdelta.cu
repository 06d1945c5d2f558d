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
constexpr int kCoef = 12;                    // numbers per token and head: beta | beta G | G | D_iC | beta D (k . k) lags 1 2 3 | - | D (k . q) lags 0 1 2 3
constexpr int kGroupsStaged = 4;             // groups per staging buffer of the scan

__device__ __forceinline__ float decay_of(float raw, float bias, float A_log) { return expf(-expf(A_log) * softplus_f(raw + bias)); }

// workspace of one group of C tokens, floats: [k: C][G N] | [q: C][G N] | [v: C][H P] | [coef: H][C][kCoef]
__host__ __device__ inline long long group_floats(int G, int H, int N, int P) { return (long long)C * (2 * G * N + H * P) + (long long)C * kCoef * H; }
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
  const int N = a.N, GN = a.G * N, HP = a.H * a.P;
  const AT* in = reinterpret_cast<const AT*>(a.in) + (long long)(s + j0) * a.ld_in;
  float* ko = a.pre + (long long)gi * group_floats(a.G, a.H, N, a.P);
  float* qo = ko + (long long)C * GN;
  float* vo = qo + (long long)C * GN;
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
    for (int n = VW * lane; n < N; n += 32 * VW) {
#pragma unroll
      for (int i = 0; i < C; ++i) {
        float k[VW], w[VW];
#pragma unroll
        for (int e = 0; e < VW; ++e) k[e] = w[e] = 0.f;
        if (i < nt) { load(in + i * a.ld_in + GN + g * N + n, k); load(in + i * a.ld_in + g * N + n, w); }
#pragma unroll
        for (int e = 0; e < VW; ++e) { k[e] *= ik[i]; w[e] *= iq[i]; }
        store(ko + (long long)i * GN + g * N + n, k); store(qo + (long long)i * GN + g * N + n, w);
      }
    }
  }
  for (int e = VW * threadIdx.x; e < C * HP; e += VW * blockDim.x) {
    const int i = e / HP;
    float v[VW];
#pragma unroll
    for (int x = 0; x < VW; ++x) v[x] = 0.f;
    if (i < nt) load(in + i * a.ld_in + 2 * GN + (e - i * HP), v);
    store(vo + e, v);
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
        if (lag > 0) { D *= gd[i - lag + 1]; o[3 + lag] = bt[i] * D * d[zk + i - lag]; }
        o[8 + lag] = D * d[zq + i - lag];
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
__device__ __forceinline__ void copy_async_4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// State in registers: L lanes share a value column, lane l holding the key rows 4 (l + L j) + e (j < NR4, e < 4), so a warp runs 32 / L columns.
// Groups arrive by asynchronous copies into one of two buffers while the buffer before is computed; rows behind N and columns behind P are
// zeros, so the loop has no bounds checks.                                    grid (B, H, ceil(P / PB)), PB = warps * 32 / L
template <int L, int NR4>
__global__ void __launch_bounds__(128) head_delta_scan_kernel(HeadDeltaArgs a) {
  constexpr int CPW = 32 / L, NP = 4 * L * NR4;
  extern __shared__ __align__(16) float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, PB = nw * CPW;
  const int l = lane % L, b = blockIdx.x, h = blockIdx.y, N = a.N, P = a.P, H = a.H, p0 = blockIdx.z * PB;
  const int g = h / (H / a.G), col = warp * CPW + lane / L, pc = p0 + col;
  const bool colok = pc < P;
  const int per = 2 * C * NP + C * PB + C * kCoef;         // floats of one group: k | q | v | coef
  const int s = a.cu[b], q = a.cu[b + 1] - s;
  if (q == 0) return;
  const bool fresh = a.ctx[b] - q == 0;
  float* gS = a.state + ((long long)a.slots[b] * H + h) * N * P + pc;
  float2 st[2 * NR4];
#pragma unroll
  for (int j = 0; j < NR4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 4 * (l + L * j) + e;
      const float v = (!fresh && colok && n < N) ? gS[(long long)n * P] : 0.f;
      if (e & 1) st[2 * j + e / 2].y = v; else st[2 * j + e / 2].x = v;
    }
  for (int e = threadIdx.x; e < 2 * kGroupsStaged * per; e += blockDim.x) smem[e] = 0.f;
  __syncthreads();
  const int GN = a.G * N, HP = H * P, vw = min(PB, P - p0), groups = (q + C - 1) / C;
  const long long gf = group_floats(a.G, H, N, P);
  const float* pre = a.pre + (long long)first_group(a.cu, b) * gf;
  const bool vec = N % 4 == 0 && P % 4 == 0 && PB % 4 == 0;          // 16-byte copies: every segment starts and ends on a 16-byte boundary
  const int n4 = vec ? N / 4 : N, v4 = vec ? vw / 4 : vw, items = C * (2 * n4 + v4) + C * kCoef / 4;
  auto fetch = [&](int g0, int ng, float* buf) {
    for (int e = threadIdx.x; e < ng * items; e += blockDim.x) {
      const int gg = e / items;
      int c = e - gg * items;
      const float* src = pre + (g0 + gg) * gf;
      float* dst = buf + gg * per;
      if (c >= C * (2 * n4 + v4)) {          // coefficients (workspace of a multiple of 4 floats in front of them or 4-byte copies)
        c -= C * (2 * n4 + v4);
        src += (long long)C * (2 * GN + HP) + (long long)h * C * kCoef + 4 * c;
        dst += 2 * C * NP + C * PB + 4 * c;
        if (vec) copy_async_16(dst, src);
        else
#pragma unroll
          for (int x = 0; x < 4; ++x) copy_async_4(dst + x, src + x);
        continue;
      }
      if (c < 2 * C * n4) {
        const int row = c / n4, x = c - row * n4;                    // row < C: keys, then queries
        src += (long long)row * GN + g * N;
        dst += row * NP;
        if (vec) copy_async_16(dst + 4 * x, src + 4 * x); else copy_async_4(dst + x, src + x);
      } else {
        c -= 2 * C * n4;
        const int row = c / v4, x = c - row * v4;
        src += (long long)2 * C * GN + (long long)row * HP + h * P + p0;
        dst += 2 * C * NP + row * PB;
        if (vec) copy_async_16(dst + 4 * x, src + 4 * x); else copy_async_4(dst + x, src + x);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, min(kGroupsStaged, groups), smem);
  int blk = 0;
  for (int g0 = 0; g0 < groups; g0 += kGroupsStaged, ++blk) {
    const int ng = min(kGroupsStaged, groups - g0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                        // these groups have landed for every thread; the other buffer is no longer read
    if (g0 + kGroupsStaged < groups) fetch(g0 + kGroupsStaged, min(kGroupsStaged, groups - g0 - kGroupsStaged), smem + ((blk + 1) & 1) * kGroupsStaged * per);
    const float* cur = smem + (blk & 1) * kGroupsStaged * per;
    for (int gg = 0; gg < ng; ++gg) {
      const float* tk = cur + gg * per;
      const float4* kq4 = reinterpret_cast<const float4*>(tk) + l;
      float2 acc[2 * C];
#pragma unroll
      for (int i = 0; i < 2 * C; ++i) acc[i] = make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < NR4; ++j)
#pragma unroll
        for (int i = 0; i < 2 * C; ++i) {
          const float4 f = kq4[i * (NP / 4) + j * L];
          acc[i] = fma2(st[2 * j], make_float2(f.x, f.y), acc[i]);
          acc[i] = fma2(st[2 * j + 1], make_float2(f.z, f.w), acc[i]);
        }
      float d[2 * C];
#pragma unroll
      for (int i = 0; i < 2 * C; ++i) d[i] = acc[i].x + acc[i].y;
      sum_over_lanes<2 * C, L>(d, lane);
      const float* vs = tk + 2 * C * NP + col;
      const float4* cf = reinterpret_cast<const float4*>(tk + 2 * C * NP + C * PB);
      float u[C], w[C], o[C], GC = 1.f;
#pragma unroll
      for (int i = 0; i < C; ++i) {
        const float4 c0 = cf[3 * i], ck = cf[3 * i + 1], cq = cf[3 * i + 2];
        float v = c0.x * vs[i * PB] - c0.y * d[i];
        if (i > 0) v -= ck.x * u[i > 0 ? i - 1 : 0];
        if (i > 1) v -= ck.y * u[i > 1 ? i - 2 : 0];
        if (i > 2) v -= ck.z * u[i > 2 ? i - 3 : 0];
        u[i] = v;
        w[i] = c0.w * v;
        float y = c0.z * d[C + i] + cq.x * v;
        if (i > 0) y += cq.y * u[i > 0 ? i - 1 : 0];
        if (i > 1) y += cq.z * u[i > 1 ? i - 2 : 0];
        if (i > 2) y += cq.w * u[i > 2 ? i - 3 : 0];
        o[i] = y;
        if (i == C - 1) GC = c0.z;
      }
#pragma unroll
      for (int j = 0; j < NR4; ++j) {
        st[2 * j] = mul2(st[2 * j], make_float2(GC, GC));
        st[2 * j + 1] = mul2(st[2 * j + 1], make_float2(GC, GC));
#pragma unroll
        for (int i = 0; i < C; ++i) {
          const float4 f = kq4[i * (NP / 4) + j * L];
          st[2 * j] = fma2(make_float2(w[i], w[i]), make_float2(f.x, f.y), st[2 * j]);
          st[2 * j + 1] = fma2(make_float2(w[i], w[i]), make_float2(f.z, f.w), st[2 * j + 1]);
        }
      }
      const int j = (g0 + gg) * C + l;       // lane l < C stores token l of the group
      const float y = l == 0 ? o[0] : l == 1 ? o[1] : l == 2 ? o[2] : o[3];
      if (l < C && colok && j < q) a.out[(long long)(s + j) * HP + h * P + pc] = y;
    }
  }
#pragma unroll
  for (int j = 0; j < NR4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 4 * (l + L * j) + e;
      if (colok && n < N) gS[(long long)n * P] = (e & 1) ? st[2 * j + e / 2].y : st[2 * j + e / 2].x;
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

template <int L>
cudaError_t scan(const HeadDeltaArgs& a, int warps, cudaStream_t s) {
  const int need = (a.N + 4 * L - 1) / (4 * L), cpw = 32 / L, PB = warps * cpw;
  auto go = [&](auto k, int nr4) -> cudaError_t {
    const size_t smem = 2 * (size_t)kGroupsStaged * (2 * C * 4 * L * nr4 + C * PB + C * kCoef) * sizeof(float);
    const cudaError_t e = allow_smem(k, smem);
    if (e != cudaSuccess) return e;
    k<<<dim3(a.B, a.H, (a.P + PB - 1) / PB), 32 * warps, smem, s>>>(a);
    return last();
  };
  if (need <= 1) return go(head_delta_scan_kernel<L, 1>, 1);
  if (need <= 2) return go(head_delta_scan_kernel<L, 2>, 2);
  if (need <= 4) return go(head_delta_scan_kernel<L, 4>, 4);
  if (need <= 8) return go(head_delta_scan_kernel<L, 8>, 8);
  return cudaErrorInvalidValue;
}

}  // namespace

bool head_delta_supported(int N) { return N >= 1 && N <= 512; }

long long head_delta_workspace(const HeadDeltaArgs& a, int max_q) {
  int vw, lw;
  return step_form(a, max_q, vw, lw) ? 0 : (long long)(a.T / C + a.B) * group_floats(a.G, a.H, a.N, a.P);
}

cudaError_t head_delta_launch(const HeadDeltaArgs& a, bool f32, int max_q, cudaStream_t s) {
  if (a.G < 1 || a.H % a.G != 0 || a.P < 1 || !head_delta_supported(a.N) || a.G > 3000) return cudaErrorInvalidValue;
  int vw, lw;
  if (step_form(a, max_q, vw, lw)) {
    if (vw == 4) AT_DISPATCH(f32, return (step<AT, 4>(a, lw, s)));
    AT_DISPATCH(f32, return (step<AT, 1>(a, lw, s)));
  }
  if (a.pre == nullptr) return cudaErrorInvalidValue;
  cudaError_t e = cudaSuccess;
  AT_DISPATCH(f32, e = prepare<AT>(a, s));
  if (e != cudaSuccess) return e;
  // few lanes per column mean few shuffles, many mean short products and more CTAs: spread while the grid leaves SMs idle
  int L = a.N <= 128 ? 4 : a.N <= 256 ? 8 : 16;
  auto ctas = [&](int lanes) { const int pb = 4 * (32 / lanes); return (long long)a.B * a.H * ((a.P + pb - 1) / pb); };
  while (L < 16 && ctas(L) < 148 && a.N > 4 * L) L *= 2;
  const int cpw = 32 / L;
  int warps = (a.P + cpw - 1) / cpw;
  if (warps > 4) warps = 4;
  return L == 4 ? scan<4>(a, warps, s) : L == 8 ? scan<8>(a, warps, s) : scan<16>(a, warps, s);
}
}  // namespace b200
