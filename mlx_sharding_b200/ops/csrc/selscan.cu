// Selective state-space scan with one step size per channel (the diagonal recurrence of a Mamba layer), the output gate included:
//   dt = softplus(dt_raw + bias),  S[c, n] <- exp(-exp(A_log[c, n]) dt_c) S[c, n] + dt_c x_c B_n,  out_c = (sum_n S[c, n] C_n + D_c x_c) silu(z_c)
//
// Conventions as in hybrid.cu: a step is a ragged batch (rows cu_seqlens[b] .. cu_seqlens[b+1] belong to sequence b, whose state lives in
// slot slots[b]; a sequence whose step starts at position 0 starts from a zero state); activations are AT = bf16 (serving) or float
// (exact mode); step sizes, decays and the state are fp32 in both.
#include "selscan.h"
#include "hybrid_common.cuh"
#include <string.h>
#include <type_traits>

namespace b200 {
namespace {

struct SelScanArgs {
  const void* x; long long ld_x;            // AT [T, I] (conv output)
  const float* dt; long long ld_dt;         // raw step sizes [T, I]
  const float* dt_bias; const float* A_log; // [I], [I, N]
  const void* bc; long long ld_bc; int b0, c0;      // AT rows with B at column b0, C at column c0
  const float* D;
  const void* gate; long long ld_g;         // AT [T, I] (nullable)
  float* state;                             // [slots, I, N]
  const int* cu; const int* ctx; const int* slots;
  void* out;                                // AT [T, I]
  int I, N, NS;
  float* ws;                                // NS > 1: per sequence [S at the step's start | end state of slices 0 .. NS-2 from a zero start: I N each | their sums of dt: I each]
};

// floats of workspace per sequence (a multiple of 4: the states are read 16 bytes at a time)
__host__ __device__ inline long long ws_stride(int I, int N, int NS) { return ((long long)NS * I * N + (long long)(NS - 1) * I + 3) / 4 * 4; }

constexpr int kCompute = 256, kHelpers = 256;       // threads of a CTA of the scan
constexpr int kStepThreads = 128;

// One step S <- exp(rate dt) S + add.  bf16 serving folds log2(e) into the rate and uses the hardware's base-2 exponential.  Exact mode adds
// S (exp(rate dt) - 1) for slow decays: a factor close to 1 would carry its last-bit error, which has a sign of its own, through every token
// of a long memory; the difference to 1 is exact to its own last bit.
template <typename AT> __device__ __forceinline__ float rate_of(float a_log);
template <> __device__ __forceinline__ float rate_of<float>(float a_log) { return -expf(a_log); }
template <> __device__ __forceinline__ float rate_of<__nv_bfloat16>(float a_log) { return -expf(a_log) * 1.4426950408889634f; }
template <typename AT> __device__ __forceinline__ float advance(float S, float rate, float dt, float x, float B);
template <> __device__ __forceinline__ float advance<float>(float S, float rate, float dt, float x, float B) {
  const float e = rate * dt;
  return e > -0.5f ? fmaf(S, expm1f(e), fmaf(x, B, S)) : fmaf(S, expf(e), x * B);
}
__device__ __forceinline__ float exp2_hw(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}
template <> __device__ __forceinline__ float advance<__nv_bfloat16>(float S, float rate, float dt, float x, float B) {
  return fmaf(exp2_hw(rate * dt), S, x * B);
}

// Step size and gate without the branches of the library's log1p and division (a helper's instructions are a dependent chain).
// softplus(v) = max(v, 0) + log1p(e), e = exp(-|v|) <= 1; log1p(e) = 2 atanh(s) with s = e / (2 + e) <= 1/3, its power series in s up to
// s^13 (the next term is below 2^-26 of the sum).
template <typename AT> __device__ __forceinline__ float step_of(float v);
template <> __device__ __forceinline__ float step_of<float>(float v) { return softplus_f(v); }
template <> __device__ __forceinline__ float step_of<__nv_bfloat16>(float v) {
  const float e = exp2_hw(-1.4426950408889634f * fabsf(v)), s = __fdividef(e, 2.f + e), z = s * s;
  float p = fmaf(z, 1.f / 13.f, 1.f / 11.f);
  p = fmaf(z, p, 1.f / 9.f);
  p = fmaf(z, p, 1.f / 7.f);
  p = fmaf(z, p, 1.f / 5.f);
  p = fmaf(z, p, 1.f / 3.f);
  return fmaxf(v, 0.f) + 2.f * fmaf(s * z, p, s);
}
template <typename AT> __device__ __forceinline__ float gated(float y, float z);
template <> __device__ __forceinline__ float gated<float>(float y, float z) { return y * silu_f(z); }
template <> __device__ __forceinline__ float gated<__nv_bfloat16>(float y, float z) {
  return y * __fdividef(z, 1.f + exp2_hw(fminf(-1.4426950408889634f * z, 126.f)));
}

// one token on SN adjacent state entries: advances S, returns the lane's part of S . C (FOLD: no output)
template <typename AT, int SN, bool FOLD>
__device__ __forceinline__ float token(float* S, const float* A, float2 ddx, const float* B, const float* C) {
  if constexpr (sizeof(AT) == 2) {
    const float2 d2 = make_float2(ddx.x, ddx.x), x2 = make_float2(ddx.y, ddx.y);
    float2 y = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < SN; i += 2) {
      const float2 r = mul2(make_float2(A[i], A[i + 1]), d2);
      const float2 xb = mul2(x2, *reinterpret_cast<const float2*>(B + i));
      const float2 s = fma2(make_float2(exp2_hw(r.x), exp2_hw(r.y)), make_float2(S[i], S[i + 1]), xb);
      S[i] = s.x; S[i + 1] = s.y;
      if (!FOLD) y = fma2(s, *reinterpret_cast<const float2*>(C + i), y);
    }
    return y.x + y.y;
  } else {
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < SN; ++i) {
      S[i] = advance<AT>(S[i], A[i], ddx.x, ddx.y, B[i]);
      if (!FOLD) y = fmaf(S[i], C[i], y);
    }
    return y;
  }
}

// SN adjacent state entries from n0 on (zeros behind N); vec: rows of a multiple of SN floats (of 4 beyond that)
template <int SN> __device__ __forceinline__ void load_states(const float* p, int n0, int N, bool vec, float* S) {
  using V = std::conditional_t<SN == 2, float2, float4>;
  constexpr int E = sizeof(V) / 4;
  if (vec) {
#pragma unroll
    for (int i = 0; i < SN; i += E) {
      V v{};
      if (n0 + i < N) v = *reinterpret_cast<const V*>(p + n0 + i);
      memcpy(S + i, &v, sizeof(V));
    }
  } else {
#pragma unroll
    for (int i = 0; i < SN; ++i) S[i] = n0 + i < N ? p[n0 + i] : 0.f;
  }
}
template <int SN> __device__ __forceinline__ void store_states(float* p, int n0, int N, bool vec, const float* S) {
  using V = std::conditional_t<SN == 2, float2, float4>;
  constexpr int E = sizeof(V) / 4;
  if (vec) {
#pragma unroll
    for (int i = 0; i < SN; i += E)
      if (n0 + i < N) { V v; memcpy(&v, S + i, sizeof(V)); *reinterpret_cast<V*>(p + n0 + i) = v; }
  } else {
#pragma unroll
    for (int i = 0; i < SN; ++i) if (n0 + i < N) p[n0 + i] = S[i];
  }
}

// the barrier both sides of a CTA arrive at (named: the two sides sit in different branches)
__device__ __forceinline__ void round_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(kCompute + kHelpers) : "memory"); }

// L lanes share a channel, lane l holding the state entries SN l .. SN l + SN - 1 in registers; a CTA runs 256 / L channels of one
// sequence (and of one time slice) with 256 compute threads, which touch shared memory only, and 256 helpers, which stage the operands of
// TOK tokens ahead (step sizes through the softplus once per channel) and finish the outputs of TOK tokens behind (D x, gate, store); both
// sides work on two buffers with one barrier per TOK tokens, and the helpers' global loads are issued one round before they are used.
// Tokens behind the end are staged as zero step sizes, which leave the state as it is.
//
// The recurrence is linear in S with a diagonal decay, so a long portion on few channels is cut into NS slices of tokens.  FOLD: the
// slice's end state from a zero start and its sum of step sizes (the product of its decays is exp(-A sum dt)) -> workspace; slice 0 also
// copies the state at the step's start there.  Main form: the start of a slice is folded from the slices before it, then its tokens run
// with outputs; the slice with the sequence's last token writes the state back.                  grid (ceil(I / channels), B, NS)
template <typename AT, int L, int SN, int TOK, bool FOLD>
__global__ void __launch_bounds__(kCompute + kHelpers, 2) selective_scan_kernel(SelScanArgs a) {
  constexpr int CPB = kCompute / L, NP = L * SN, EPT = (TOK * CPB + kHelpers - 1) / kHelpers, BPT = (TOK * NP + kHelpers - 1) / kHelpers;
  __shared__ __align__(16) float Bs[2][TOK * NP];
  __shared__ __align__(16) float Cs[FOLD ? 1 : 2][FOLD ? 4 : TOK * NP];
  __shared__ __align__(16) float2 ds[2][TOK * CPB];         // (dt, dt x)
  __shared__ __align__(16) float ys[FOLD ? 1 : 2][FOLD ? 4 : TOK * CPB];
  const int b = blockIdx.y, sl = blockIdx.z, I = a.I, N = a.N, NS = a.NS, c_0 = blockIdx.x * CPB;
  const int s = a.cu[b], q = a.cu[b + 1] - s;
  if (q == 0) return;
  const int len = (q + NS - 1) / NS, j_0 = sl * len, j_1 = min(q, j_0 + len);
  if (j_0 >= j_1) return;
  const int tiles = (j_1 - j_0 + TOK - 1) / TOK;
  const long long IN = (long long)I * N;
  float* ws = a.ws + b * ws_stride(I, N, NS);
  if (threadIdx.x >= kCompute) {
    // ---- helpers
    if (FOLD && j_1 == q) return;             // nothing follows this slice (the compute threads leave as well, before any barrier)
    const int tid = threadIdx.x - kCompute;
    const AT* X = reinterpret_cast<const AT*>(a.x);
    const AT* BC = reinterpret_cast<const AT*>(a.bc);
    const AT* Z = reinterpret_cast<const AT*>(a.gate);
    // operands in flight, as they are stored: addresses behind the end are clamped and the values dropped when they are used, so that no
    // load waits for another's conversion
    float rd[EPT], bias[EPT], Dk[EPT];
    AT rx[EPT], rb[BPT], rc[BPT], ex[EPT], ez[EPT];
#pragma unroll
    for (int i = 0; i < EPT; ++i) {
      const int k = c_0 + (tid + i * kHelpers) % CPB;
      bias[i] = k < I ? a.dt_bias[k] : 0.f;
      Dk[i] = !FOLD && k < I ? a.D[k] : 0.f;
    }
    auto fetch = [&](int tile) {    // operands of a tile -> registers
#pragma unroll
      for (int i = 0; i < EPT; ++i) {
        const int e = tid + i * kHelpers, j = min(j_0 + tile * TOK + e / CPB, j_1 - 1), k = min(c_0 + e % CPB, I - 1);
        rd[i] = a.dt[(long long)(s + j) * a.ld_dt + k];
        rx[i] = X[(long long)(s + j) * a.ld_x + k];
      }
#pragma unroll
      for (int i = 0; i < BPT; ++i) {
        const int e = tid + i * kHelpers, j = min(j_0 + tile * TOK + e / NP, j_1 - 1), n = min(e % NP, N - 1);
        const AT* row = BC + (long long)(s + j) * a.ld_bc + n;
        rb[i] = row[a.b0];
        if (!FOLD) rc[i] = row[a.c0];
      }
    };
    auto stage = [&](int tile) {
#pragma unroll
      for (int i = 0; i < EPT; ++i) {
        const int e = tid + i * kHelpers;
        const bool ok = j_0 + tile * TOK + e / CPB < j_1 && c_0 + e % CPB < I;
        const float d = ok ? step_of<AT>(rd[i] + bias[i]) : 0.f;
        if (TOK * CPB % kHelpers == 0 || e < TOK * CPB) ds[tile & 1][e] = make_float2(d, d * ldf<AT>(&rx[i]));
      }
#pragma unroll
      for (int i = 0; i < BPT; ++i) {
        const int e = tid + i * kHelpers;
        const bool ok = e % NP < N;
        if (TOK * NP % kHelpers == 0 || e < TOK * NP) {
          Bs[tile & 1][e] = ok ? ldf<AT>(&rb[i]) : 0.f;
          if (!FOLD) Cs[tile & 1][e] = ok ? ldf<AT>(&rc[i]) : 0.f;
        }
      }
    };
    auto fetch_out = [&](int tile) {        // x and gate of a tile whose outputs are finished later
#pragma unroll
      for (int i = 0; i < EPT; ++i) {
        const int e = tid + i * kHelpers, j = min(j_0 + tile * TOK + e / CPB, j_1 - 1), k = min(c_0 + e % CPB, I - 1);
        ex[i] = X[(long long)(s + j) * a.ld_x + k];
        if (Z != nullptr) ez[i] = Z[(long long)(s + j) * a.ld_g + k];
      }
    };
    auto finish = [&](int tile) {
#pragma unroll
      for (int i = 0; i < EPT; ++i) {
        const int e = tid + i * kHelpers, j = j_0 + tile * TOK + e / CPB, k = c_0 + e % CPB;
        if (e >= TOK * CPB || j >= j_1 || k >= I) continue;
        float y = ys[tile & 1][e] + Dk[i] * ldf<AT>(&ex[i]);
        if (Z != nullptr) y = gated<AT>(y, ldf<AT>(&ez[i]));
        stf<AT>((AT*)a.out + (long long)(s + j) * I + k, y);
      }
    };
    fetch(0);
    stage(0);
    fetch(1);
    round_barrier();
    for (int k = 0; k < tiles; ++k) {         // round k: tile k is computed
      if (k + 1 < tiles) stage(k + 1);
      if (k + 2 < tiles) fetch(k + 2);
      if (!FOLD) {
        if (k > 0) finish(k - 1);
        fetch_out(k);
      }
      round_barrier();
    }
    if (!FOLD) finish(tiles - 1);
    return;
  }
  // ---- compute threads
  const int ch = threadIdx.x / L, l = threadIdx.x % L, c = c_0 + ch, n0 = l * SN;
  const bool fresh = a.ctx[b] - q == 0, live = c < I, vec = N % (SN == 2 ? 2 : 4) == 0;
  const int cc = live ? c : 0;
  float S[SN], A[SN];
  float* gS = a.state + ((long long)a.slots[b] * I + cc) * N;
  float* wS = ws + (long long)cc * N;       // + i * IN: start state (i = 0), end state of slice i - 1
  float* wd = ws + NS * IN + cc;            // + i * I: sum of the step sizes of slice i
  if (fresh && (NS == 1 || FOLD)) {
#pragma unroll
    for (int i = 0; i < SN; ++i) S[i] = 0.f;
  } else {
    load_states<SN>(NS == 1 || FOLD ? gS : wS, n0, N, vec, S);
  }
  load_states<SN>(a.A_log + (long long)cc * N, n0, N, vec, A);
#pragma unroll
  for (int i = 0; i < SN; ++i) A[i] = n0 + i < N ? rate_of<AT>(A[i]) : 0.f;
  if (FOLD) {
    if (sl == 0 && live) store_states<SN>(wS, n0, N, vec, S);
    if (j_1 == q) return;
#pragma unroll
    for (int i = 0; i < SN; ++i) S[i] = 0.f;
  } else {
    for (int k = 0; k < sl; ++k) {
      float E[SN];
      load_states<SN>(wS + (k + 1) * IN, n0, N, vec, E);
      const float d = wd[(long long)k * I];
#pragma unroll
      for (int i = 0; i < SN; ++i) S[i] = advance<AT>(S[i], A[i], d, 1.f, E[i]);
    }
  }
  float sum_dt = 0.f;
  round_barrier();
  for (int k = 0; k < tiles; ++k) {
    const int buf = k & 1;
    const float2* dk = ds[buf] + ch;
    const float* Bk = Bs[buf] + n0;
    const float* Ck = FOLD ? Bk : Cs[FOLD ? 0 : buf] + n0;
#pragma unroll 2
    for (int j = 0; j < TOK; j += 4) {
      float y[4];
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        const float2 d = dk[(j + t) * CPB];
        y[t] = token<AT, SN, FOLD>(S, A, d, Bk + (j + t) * NP, Ck + (j + t) * NP);
        if (FOLD) sum_dt += d.x;
      }
      if (FOLD) continue;
      // sums over the L lanes of a channel, four tokens at once: after the first two levels lane l holds token l % 4
      float* yk = ys[FOLD ? 0 : buf] + j * CPB + ch;
      if (L == 1) {
#pragma unroll
        for (int t = 0; t < 4; ++t) yk[t * CPB] = y[t];
      } else {
        const bool odd = l & 1;
        const float u0 = (odd ? y[1] : y[0]) + __shfl_xor_sync(0xffffffffu, odd ? y[0] : y[1], 1);
        const float u1 = (odd ? y[3] : y[2]) + __shfl_xor_sync(0xffffffffu, odd ? y[2] : y[3], 1);
        if (L == 2) {
          yk[(odd ? 1 : 0) * CPB] = u0; yk[(odd ? 3 : 2) * CPB] = u1;
        } else {
          const bool hi = l & 2;
          float v = (hi ? u1 : u0) + __shfl_xor_sync(0xffffffffu, hi ? u0 : u1, 2);
#pragma unroll
          for (int o = 4; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
          if (L == 4 || l < 4) yk[(l & 3) * CPB] = v;
        }
      }
    }
    round_barrier();
  }
  if (!live) return;
  if (FOLD) {
    store_states<SN>(wS + (long long)(sl + 1) * IN, n0, N, vec, S);
    if (l == 0) wd[(long long)sl * I] = sum_dt;
  } else if (j_1 == q) {
    store_states<SN>(gS, n0, N, vec, S);
  }
}

// One token per sequence (decode): no staging, every operand straight into registers, kStepSeqs sequences per thread so that their state
// loads are in flight together and the rates are computed once.                        grid (ceil(I / channels), ceil(B / kStepSeqs))
constexpr int kStepSeqs = 4;

template <typename AT, int L, int SN>
__global__ void __launch_bounds__(kStepThreads) selective_step_kernel(SelScanArgs a, int B) {
  constexpr int CPB = kStepThreads / L;
  const int I = a.I, N = a.N, l = threadIdx.x % L, c = blockIdx.x * CPB + threadIdx.x / L, n0 = l * SN;
  const bool live = c < I, vec = N % (SN == 2 ? 2 : 4) == 0;
  const int cc = live ? c : 0;
  float S[kStepSeqs][SN], A[SN], d[kStepSeqs];
  AT Bv[kStepSeqs][SN], Cv[kStepSeqs][SN], x[kStepSeqs], z[kStepSeqs];         // as they are stored: no load waits for another's conversion
  float* gS[kStepSeqs];
  bool on[kStepSeqs], fresh[kStepSeqs];
  long long row[kStepSeqs];
  const AT* X = reinterpret_cast<const AT*>(a.x);
  const AT* BC = reinterpret_cast<const AT*>(a.bc);
  const AT* Z = reinterpret_cast<const AT*>(a.gate);
#pragma unroll
  for (int i = 0; i < kStepSeqs; ++i) {       // behind the end: the last sequence, never stored
    const int b = min(blockIdx.y * kStepSeqs + i, B - 1), t0 = a.cu[b], t1 = a.cu[b + 1];
    on[i] = blockIdx.y * kStepSeqs + i < B && t1 > t0;
    row[i] = min(t0, a.cu[B] - 1);
    fresh[i] = a.ctx[b] == 1;                 // the sequence's first token
    gS[i] = a.state + ((long long)a.slots[b] * I + cc) * N;
  }
#pragma unroll
  for (int i = 0; i < kStepSeqs; ++i) {
    load_states<SN>(gS[i], n0, N, vec, S[i]);
    d[i] = a.dt[row[i] * a.ld_dt + cc];
    x[i] = X[row[i] * a.ld_x + cc];
    if (Z != nullptr) z[i] = Z[row[i] * a.ld_g + cc];
    const AT* p = BC + row[i] * a.ld_bc;
#pragma unroll
    for (int k = 0; k < SN; ++k) { const int n = min(n0 + k, N - 1); Bv[i][k] = p[a.b0 + n]; Cv[i][k] = p[a.c0 + n]; }
  }
  load_states<SN>(a.A_log + (long long)cc * N, n0, N, vec, A);
  const float bias = a.dt_bias[cc], Dk = a.D[cc];
#pragma unroll
  for (int k = 0; k < SN; ++k) A[k] = n0 + k < N ? rate_of<AT>(A[k]) : 0.f;
#pragma unroll
  for (int i = 0; i < kStepSeqs; ++i) {
    if (!on[i]) continue;                     // uniform over the CTA
    const float dt = step_of<AT>(d[i] + bias), xv = ldf<AT>(&x[i]);
    float y = 0.f;
#pragma unroll
    for (int k = 0; k < SN; ++k) {
      S[i][k] = advance<AT>(fresh[i] ? 0.f : S[i][k], A[k], dt, dt * xv, n0 + k < N ? ldf<AT>(&Bv[i][k]) : 0.f);
      y = fmaf(S[i][k], n0 + k < N ? ldf<AT>(&Cv[i][k]) : 0.f, y);
    }
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!live) continue;
    store_states<SN>(gS[i], n0, N, vec, S[i]);
    if (l == 0) {
      y += Dk * xv;
      if (Z != nullptr) y = gated<AT>(y, ldf<AT>(&z[i]));
      stf<AT>((AT*)a.out + row[i] * I + c, y);
    }
  }
}

// lanes per channel and state entries per lane: of the scan (two entries per lane while a warp covers the state: a token's instructions
// are a dependent chain, more warps hide it) and of the step kernel (16 bytes of state per load)
struct ScanShape { int L, SN; };
ScanShape scan_shape(int N, int SN) {
  ScanShape r{1, SN};
  while (r.L < 32 && r.L * r.SN < N) r.L *= 2;
  while (r.L * r.SN < N) r.SN *= 2;
  return r;
}

template <typename AT, int L, int SN>
cudaError_t scan_t(const SelScanArgs& a, int B, cudaStream_t s) {
  constexpr int CPB = kCompute / L, TOK = L <= 2 ? 4 : L == 4 ? 8 : L == 8 ? 32 : L * SN <= 64 ? 16 : L * SN <= 128 ? 8 : 4;
  const dim3 grid((a.I + CPB - 1) / CPB, B, a.NS);
  if (a.NS > 1) selective_scan_kernel<AT, L, SN, TOK, true><<<grid, kCompute + kHelpers, 0, s>>>(a);
  selective_scan_kernel<AT, L, SN, TOK, false><<<grid, kCompute + kHelpers, 0, s>>>(a);
  return last();
}

template <typename AT, int L, int SN>
cudaError_t step_t(const SelScanArgs& a, int B, cudaStream_t s) {
  constexpr int CPB = kStepThreads / L;
  selective_step_kernel<AT, L, SN><<<dim3((a.I + CPB - 1) / CPB, (B + kStepSeqs - 1) / kStepSeqs), kStepThreads, 0, s>>>(a, B);
  return last();
}

}  // namespace

bool selective_scan_supported(int N) { return N >= 1 && N <= 256; }

// Two passes over NS slices take about 2 / NS of the time of one pass while there are idle SMs: worth it from four slices on.
int selective_scan_slices(int B, int I, int N, int max_q) {
  const int cpb = kCompute / scan_shape(N, 2).L;
  const long long ctas = (long long)B * ((I + cpb - 1) / cpb);
  int ns = 1;
  while (ns < 32 && ctas * ns * 2 <= 296 && max_q >= 128 * ns) ns *= 2;       // slices of at least 64 tokens
  return ns >= 4 ? ns : 1;
}

long long selective_scan_workspace(int B, int I, int N, int slices) {
  return slices > 1 ? B * ws_stride(I, N, slices) : 0;
}

cudaError_t selective_scan_launch(const void* x, long long ld_x, const float* dt, long long ld_dt, const float* dt_bias, const float* A_log, const void* bc,
                                  long long ld_bc, int b0, int c0, const float* D, const void* gate, long long ld_g, float* state, const int* cu,
                                  const int* ctx, const int* slots, void* out, int B, int I, int N, bool f32, int max_q, int slices, float* ws,
                                  cudaStream_t s) {
  if (!selective_scan_supported(N) || slices < 1 || (slices > 1 && ws == nullptr)) return cudaErrorInvalidValue;
  const SelScanArgs a{x, ld_x, dt, ld_dt, dt_bias, A_log, bc, ld_bc, b0, c0, D, gate, ld_g, state, cu, ctx, slots, out, I, N, slices, ws};
#define SCAN_CASE(F, LL, NN) if (sh.L == LL && sh.SN == NN) AT_DISPATCH(f32, return (F<AT, LL, NN>(a, B, s)))
  if (max_q <= 1) {
    const ScanShape sh = scan_shape(N, 4);
    SCAN_CASE(step_t, 1, 4); SCAN_CASE(step_t, 2, 4); SCAN_CASE(step_t, 4, 4); SCAN_CASE(step_t, 8, 4); SCAN_CASE(step_t, 16, 4); SCAN_CASE(step_t, 32, 4);
    SCAN_CASE(step_t, 32, 8);
  } else {
    const ScanShape sh = scan_shape(N, 2);
    SCAN_CASE(scan_t, 1, 2); SCAN_CASE(scan_t, 2, 2); SCAN_CASE(scan_t, 4, 2); SCAN_CASE(scan_t, 8, 2); SCAN_CASE(scan_t, 16, 2); SCAN_CASE(scan_t, 32, 2);
    SCAN_CASE(scan_t, 32, 4); SCAN_CASE(scan_t, 32, 8);
  }
#undef SCAN_CASE
  return cudaErrorInvalidValue;
}
}  // namespace b200
