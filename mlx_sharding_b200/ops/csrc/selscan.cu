// Selective state-space scan with one step size per channel (the diagonal recurrence of a Mamba layer), the output gate included:
//   dt = softplus(dt_raw + bias),  S[c, n] <- exp(-exp(A_log[c, n]) dt_c) S[c, n] + dt_c x_c B_n,  out_c = (sum_n S[c, n] C_n + D_c x_c) silu(z_c)
//
// Conventions as in hybrid.cu: a step is a ragged batch (rows cu_seqlens[b] .. cu_seqlens[b+1] belong to sequence b, whose state lives in
// slot slots[b]; a sequence whose step starts at position 0 starts from a zero state); activations are AT = bf16 (serving) or float
// (exact mode); step sizes, decays and the state are fp32 in both.
#include "selscan.h"
#include "hybrid_common.cuh"

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

constexpr int kScanThreads = 128;
constexpr int kScanTokens = 16;             // tokens staged in shared memory at a time

// decay factors: the exact path calls expf; bf16 serving folds log2(e) into the rate and uses the hardware's base-2 exponential
template <typename AT> __device__ __forceinline__ float rate_of(float a_log);
template <> __device__ __forceinline__ float rate_of<float>(float a_log) { return -expf(a_log); }
template <> __device__ __forceinline__ float rate_of<__nv_bfloat16>(float a_log) { return -expf(a_log) * 1.4426950408889634f; }
template <typename AT> __device__ __forceinline__ float decay_of(float rate, float dt);
template <> __device__ __forceinline__ float decay_of<float>(float rate, float dt) { return expf(rate * dt); }
template <> __device__ __forceinline__ float decay_of<__nv_bfloat16>(float rate, float dt) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(rate * dt));
  return r;
}

template <int SN> __device__ __forceinline__ void load_states(const float* p, int n0, int N, bool vec, float* S) {
  if (vec) {
#pragma unroll
    for (int i = 0; i < SN; i += 4) {
      const float4 v = n0 + i < N ? *reinterpret_cast<const float4*>(p + n0 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < SN; ++i) S[i] = n0 + i < N ? p[n0 + i] : 0.f;
  }
}
template <int SN> __device__ __forceinline__ void store_states(float* p, int n0, int N, bool vec, const float* S) {
  if (vec) {
#pragma unroll
    for (int i = 0; i < SN; i += 4)
      if (n0 + i < N) *reinterpret_cast<float4*>(p + n0 + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < SN; ++i) if (n0 + i < N) p[n0 + i] = S[i];
  }
}

// L lanes share a channel, lane l holding the state entries SN l .. SN l + SN - 1 in registers; a CTA runs kScanThreads / L channels of one
// sequence (and of one time slice).  The operands of kTok tokens are staged in shared memory as floats (step sizes through the softplus
// once per channel); the outputs go back through shared memory so that gate and store are coalesced.
//
// The recurrence is linear in S with a diagonal decay, so a long portion is cut into NS slices of tokens.  FOLD: the slice's end state from
// a zero start and its sum of step sizes (the product of its decays is exp(-A sum dt)) -> workspace; slice 0 also copies the state at the
// step's start there.  Main form: the start of a slice is folded from the slices before it, then its tokens run with outputs; the slice
// with the sequence's last token writes the state back.                    grid (ceil(I / channels), B, NS)
template <typename AT, int L, int SN, bool FOLD>
__global__ void __launch_bounds__(kScanThreads) selective_scan_kernel(SelScanArgs a, int kTok) {
  constexpr int CPB = kScanThreads / L, NP = L * SN;
  extern __shared__ __align__(16) float smem[];
  float* Bs = smem;                         // [tok][NP]
  float* Cs = Bs + kTok * NP;               // [tok][NP]
  float* ds = Cs + kTok * NP;               // [tok][CPB]
  float* xs = ds + kTok * CPB;              // [tok][CPB]
  float* ys = xs + kTok * CPB;              // [tok][CPB]
  const int b = blockIdx.y, sl = blockIdx.z, I = a.I, N = a.N, NS = a.NS;
  const int c_0 = blockIdx.x * CPB, ch = threadIdx.x / L, l = threadIdx.x % L, c = c_0 + ch, n0 = l * SN;
  const int s = a.cu[b], q = a.cu[b + 1] - s;
  if (q == 0) return;
  const int len = (q + NS - 1) / NS, j_0 = sl * len, j_1 = min(q, j_0 + len);
  if (j_0 >= j_1) return;
  const bool fresh = a.ctx[b] - q == 0, live = c < I, vec = N % 4 == 0;
  const int cc = live ? c : 0;
  float S[SN], A[SN];
  float* gS = a.state + ((long long)a.slots[b] * I + cc) * N;
  const long long IN = (long long)I * N;
  float* ws = a.ws + b * ws_stride(I, N, NS);
  float* wS = ws + (long long)cc * N;       // + i * IN: start state (i = 0), end state of slice i - 1
  float* wd = ws + NS * IN + cc;            // + i * I: sum of the step sizes of slice i
  if (NS == 1 || FOLD) {
    if (fresh) {
#pragma unroll
      for (int i = 0; i < SN; ++i) S[i] = 0.f;
    } else {
      load_states<SN>(gS, n0, N, vec, S);
    }
  } else {
    load_states<SN>(wS, n0, N, vec, S);
  }
  load_states<SN>(a.A_log + (long long)cc * N, n0, N, vec, A);
#pragma unroll
  for (int i = 0; i < SN; ++i) A[i] = n0 + i < N ? rate_of<AT>(A[i]) : 0.f;
  if (FOLD) {
    if (sl == 0 && live) store_states<SN>(wS, n0, N, vec, S);
    if (j_1 == q) return;                   // nothing follows this slice
#pragma unroll
    for (int i = 0; i < SN; ++i) S[i] = 0.f;
  } else {
    for (int k = 0; k < sl; ++k) {
      float E[SN];
      load_states<SN>(wS + (k + 1) * IN, n0, N, vec, E);
      const float d = wd[(long long)k * I];
#pragma unroll
      for (int i = 0; i < SN; ++i) S[i] = decay_of<AT>(A[i], d) * S[i] + E[i];
    }
  }
  float sum_dt = 0.f;
  const AT* X = reinterpret_cast<const AT*>(a.x);
  const AT* BC = reinterpret_cast<const AT*>(a.bc);
  for (int jb = j_0; jb < j_1; jb += kTok) {
    const int nt = min(kTok, j_1 - jb);
    const long long t0 = s + jb;
    __syncthreads();                        // the last tokens' operands and outputs are no longer read
#pragma unroll 4
    for (int e = threadIdx.x; e < nt * CPB; e += kScanThreads) {
      const int jj = e / CPB, k = c_0 + e % CPB;
      float d = 0.f, xv = 0.f;
      if (k < I) {
        d = softplus_f(a.dt[(t0 + jj) * a.ld_dt + k] + a.dt_bias[k]);
        xv = ldf<AT>(X + (t0 + jj) * a.ld_x + k);
      }
      ds[e] = d; xs[e] = xv;
    }
#pragma unroll 2
    for (int e = threadIdx.x; e < nt * NP; e += kScanThreads) {
      const int jj = e / NP, n = e % NP;
      const AT* row = BC + (t0 + jj) * a.ld_bc;
      Bs[e] = n < N ? ldf<AT>(row + a.b0 + n) : 0.f;
      if (!FOLD) Cs[e] = n < N ? ldf<AT>(row + a.c0 + n) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int jj = 0; jj < nt; ++jj) {
      const float d = ds[jj * CPB + ch], dx = d * xs[jj * CPB + ch];
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < SN; i += 4) {
        const float4 B4 = *reinterpret_cast<const float4*>(Bs + jj * NP + n0 + i);
        S[i] = decay_of<AT>(A[i], d) * S[i] + dx * B4.x;
        S[i + 1] = decay_of<AT>(A[i + 1], d) * S[i + 1] + dx * B4.y;
        S[i + 2] = decay_of<AT>(A[i + 2], d) * S[i + 2] + dx * B4.z;
        S[i + 3] = decay_of<AT>(A[i + 3], d) * S[i + 3] + dx * B4.w;
        if (!FOLD) {
          const float4 C4 = *reinterpret_cast<const float4*>(Cs + jj * NP + n0 + i);
          y += S[i] * C4.x + S[i + 1] * C4.y + S[i + 2] * C4.z + S[i + 3] * C4.w;
        }
      }
      if (FOLD) {
        sum_dt += d;
      } else {
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        if (l == 0) ys[jj * CPB + ch] = y;
      }
    }
    if (FOLD) continue;
    __syncthreads();
#pragma unroll 4
    for (int e = threadIdx.x; e < nt * CPB; e += kScanThreads) {
      const int jj = e / CPB, k = c_0 + e % CPB;
      if (k >= I) continue;
      float y = ys[e] + a.D[k] * xs[e];
      if (a.gate != nullptr) y *= silu_f(ldf<AT>((const AT*)a.gate + (t0 + jj) * a.ld_g + k));
      stf<AT>((AT*)a.out + (t0 + jj) * I + k, y);
    }
  }
  if (!live) return;
  if (FOLD) {
    store_states<SN>(wS + (long long)(sl + 1) * IN, n0, N, vec, S);
    if (l == 0) wd[(long long)sl * I] = sum_dt;
  } else if (j_1 == q) {
    store_states<SN>(gS, n0, N, vec, S);
  }
}

struct ScanShape { int L, SN; };
ScanShape scan_shape(int N) {
  ScanShape r{1, 4};
  while (r.L < 32 && r.L * r.SN < N) r.L *= 2;
  if (r.L * r.SN < N) r.SN = 8;
  return r;
}

}  // namespace

bool selective_scan_supported(int N) { return N >= 1 && N <= 256; }

int selective_scan_slices(int B, int I, int N, int max_q) {
  const int cpb = kScanThreads / scan_shape(N).L;
  const long long ctas = (long long)B * ((I + cpb - 1) / cpb);
  int ns = 1;
  while (ns < 32 && ctas * ns < 592 && max_q >= 128 * ns) ns *= 2;       // slices of at least 64 tokens
  return ns;
}

long long selective_scan_workspace(int B, int I, int N, int slices) {
  return slices > 1 ? B * ws_stride(I, N, slices) : 0;
}

cudaError_t selective_scan_launch(const void* x, long long ld_x, const float* dt, long long ld_dt, const float* dt_bias, const float* A_log, const void* bc,
                                  long long ld_bc, int b0, int c0, const float* D, const void* gate, long long ld_g, float* state, const int* cu,
                                  const int* ctx, const int* slots, void* out, int B, int I, int N, bool f32, int max_q, int slices, float* ws,
                                  cudaStream_t s) {
  if (!selective_scan_supported(N) || slices < 1 || (slices > 1 && ws == nullptr)) return cudaErrorInvalidValue;
  SelScanArgs a{x, ld_x, dt, ld_dt, dt_bias, A_log, bc, ld_bc, b0, c0, D, gate, ld_g, state, cu, ctx, slots, out, I, N, slices, ws};
  const ScanShape sh = scan_shape(N);
  const int cpb = kScanThreads / sh.L, tok = max_q < 1 ? 1 : (max_q < kScanTokens ? max_q : kScanTokens);
  const size_t smem = (size_t)tok * (2 * sh.L * sh.SN + 3 * cpb) * sizeof(float);
  const dim3 grid((I + cpb - 1) / cpb, B, slices);
  auto go = [&](auto fold, auto run) -> cudaError_t {
    if (slices > 1) fold<<<grid, kScanThreads, smem, s>>>(a, tok);
    run<<<grid, kScanThreads, smem, s>>>(a, tok);
    return last();
  };
#define SCAN_CASE(LL, NN) \
  if (sh.L == LL && sh.SN == NN) { AT_DISPATCH(f32, return go(selective_scan_kernel<AT, LL, NN, true>, selective_scan_kernel<AT, LL, NN, false>)); }
  SCAN_CASE(1, 4) SCAN_CASE(2, 4) SCAN_CASE(4, 4) SCAN_CASE(8, 4) SCAN_CASE(16, 4) SCAN_CASE(32, 4) SCAN_CASE(32, 8)
#undef SCAN_CASE
  return cudaErrorInvalidValue;
}
}  // namespace b200
