// Kernels of stacks that run on several residual streams with dynamic-tanh norms: the stream update fused with the read for the next
// sublayer, the gated delta rule with one decay per head and key channel, the prologue of grouped-query attention (per-head RMS norm of
// queries and keys, rotation, value mixing, append to the paged pools; the attention itself is in sinkattn.cu), minGRU, the group-limited
// softmax router and the squared ReLU.
//
// Conventions as in hybrid.cu: a step is a ragged batch (rows cu_seqlens[b] .. cu_seqlens[b+1] belong to sequence b, whose recurrent
// state lives in slot slots[b]; a sequence whose step starts at position 0 starts from a zero state); activations are AT = bf16
// (serving) or float (exact mode); streams, norms, scores, softmax, router and everything inside a recurrence are fp32 in both.
#include "streams.h"
#include "hybrid_common.cuh"

namespace b200 {
namespace {

constexpr int kMaxStreams = 8;

// ---------------------------------------------------------------------------------------------------------- streams
// xs[t, s, :] = table[ids[t], :] * scale (+ pos[positions[t], :], pos nullable) for every stream s
template <typename TT>
__global__ void stream_embed_kernel(const TT* __restrict__ table, long long ld, const long long* __restrict__ ids, float scale, int S, int n,
                                    float* __restrict__ xs, const TT* __restrict__ pos, const int* __restrict__ positions, int n_pos) {
  const long long t = blockIdx.x;
  const TT* row = table + ids[t] * ld;
  const TT* prow = pos != nullptr ? pos + (long long)min(max(positions[t], 0), n_pos - 1) * n : nullptr;      // (the host admits no position behind the table)
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < n; c += gridDim.y * blockDim.x) {
    float v = ldf<TT>(row + c) * scale;
    if (prow != nullptr) v += ldf<TT>(prow + c);
    for (int s = 0; s < S; ++s) xs[(t * S + s) * n + c] = v;
  }
}

struct HyperArgs {
  float* xs;                                // [T, S, n] fp32, updated in place
  const float* y; long long ld_y;           // sublayer output (nullptr: only the read)
  const float* y2; long long ld_y2;         // second branch added to y (nullable)
  const void* gate; long long ld_g;         // gate logits per element, AT (nullable)
  const float* ls;                          // [n] layer scale (nullable)
  const float* mix; const float* out_w;     // [S, S] (from, to), [S]
  const float* in_w;                        // [S] weights of the read that follows
  const float* w; const float* b;           // dynamic tanh of the read: tanh(alpha u) * w + b
  float mult, alpha;
  void* xa;                                 // AT [T, n]
  int S, n;
};

// r = (y + y2) * ls * sigmoid(gate);  xs[t, j] <- sum_s mix[s, j] xs[t, s] + mult * out_w[j] * r;  xa = dyt(sum_j in_w[j] xs[t, j]).
// No row statistics anywhere: every (token, channel) is independent.                      grid (T, ceil(n / blockDim))
template <typename AT>
__global__ void hyper_step_kernel(HyperArgs a) {
  __shared__ float sm[kMaxStreams * kMaxStreams + 2 * kMaxStreams];
  const int S = a.S;
  float* mix = sm; float* ow = sm + kMaxStreams * kMaxStreams; float* iw = ow + kMaxStreams;
  if (threadIdx.x < S * S && a.y != nullptr) mix[threadIdx.x] = a.mix[threadIdx.x];
  if (threadIdx.x < S) { ow[threadIdx.x] = a.y != nullptr ? a.mult * a.out_w[threadIdx.x] : 0.f; iw[threadIdx.x] = a.in_w[threadIdx.x]; }
  __syncthreads();
  const long long t = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= a.n) return;
  float* x = a.xs + t * S * a.n + c;
  float old[kMaxStreams], u = 0.f;
#pragma unroll
  for (int s = 0; s < kMaxStreams; ++s) old[s] = s < S ? x[(long long)s * a.n] : 0.f;
  if (a.y != nullptr) {
    float r = a.y[t * a.ld_y + c];
    if (a.y2 != nullptr) r += a.y2[t * a.ld_y2 + c];
    if (a.ls != nullptr) r *= a.ls[c];
    if (a.gate != nullptr) r *= sigmoid_f(ldf<AT>((const AT*)a.gate + t * a.ld_g + c));
#pragma unroll
    for (int j = 0; j < kMaxStreams; ++j) {
      if (j < S) {
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < kMaxStreams; ++s) if (s < S) v += mix[s * S + j] * old[s];
        v += ow[j] * r;
        x[(long long)j * a.n] = v;
        u += iw[j] * v;
      }
    }
  } else {
#pragma unroll
    for (int j = 0; j < kMaxStreams; ++j) if (j < S) u += iw[j] * old[j];
  }
  stf<AT>((AT*)a.xa + t * a.n + c, tanhf(a.alpha * u) * a.w[c] + a.b[c]);
}

template <typename AT>
__global__ void relu2_kernel(AT* __restrict__ x, long long ld, int n) {
  AT* row = x + (long long)blockIdx.x * ld;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < n; c += gridDim.y * blockDim.x) {
    const float v = fmaxf(ldf<AT>(row + c), 0.f);
    stf<AT>(row + c, v * v);
  }
}

// ---------------------------------------------------------------------------------------------------------- gated delta rule
struct DeltaArgs {
  const void* in; long long ld_in;          // conv output, AT: [q: G*N | k: G*N | v: H*P]
  const void* beta; long long ld_b;         // raw write strengths, AT [T, >= H]
  const float* dt; long long ld_dt;         // raw step sizes fp32 [T, H*N]
  const float* dt_bias; const float* A_log; // [H*N], [H]
  float* state;                             // [slots, H, N, P]
  const int* cu; const int* ctx; const int* slots;
  float* out;                               // fp32 [T, H*P]
  int H, G, N, P;
  float q_scale, unit_eps;
  const float* pre; long long ld_pre;       // register form only: fp32 rows [k unit | q unit * q_scale | decay | v | sigmoid(beta)] (delta_prepare_kernel)
};

// Operands of `nt` tokens (rows t0 ..) of head h for a delta-rule CTA: kq[jj] = [k unit | q unit * q_scale | decay], each `ldn` >= N
// floats wide (zeros behind N), vs[jj] = the CTA's PB value columns (zeros behind the head's last column), bs[jj] = sigmoid(beta).
// All threads load element-wise (independent loads), then one warp per token takes the two sums of squares from shared memory and
// rescales.  Ends with a barrier.
template <typename AT>
__device__ __forceinline__ void delta_stage(const DeltaArgs& a, long long t0, int nt, int h, int g, int p0, int PB, float negA, float* kq, float* vs,
                                            float* bs, int ldn) {
  const int N = a.N, GN = a.G * N, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const AT* in = reinterpret_cast<const AT*>(a.in);
#pragma unroll 4
  for (int e = threadIdx.x; e < nt * ldn; e += blockDim.x) {
    const int jj = e / ldn, n = e - jj * ldn;
    float* dst = kq + jj * 3 * ldn;
    float kv = 0.f, qv = 0.f, gv = 0.f;
    if (n < N) {
      const AT* row = in + (t0 + jj) * a.ld_in;
      kv = ldf<AT>(row + GN + g * N + n);
      qv = ldf<AT>(row + g * N + n);
      gv = expf(negA * softplus_f(a.dt[(t0 + jj) * a.ld_dt + h * N + n] + a.dt_bias[h * N + n]));
    }
    dst[n] = kv; dst[ldn + n] = qv; dst[2 * ldn + n] = gv;
  }
#pragma unroll 2
  for (int e = threadIdx.x; e < nt * PB; e += blockDim.x) {
    const int jj = e / PB, c = e - jj * PB;
    vs[e] = p0 + c < a.P ? ldf<AT>(in + (t0 + jj) * a.ld_in + 2 * GN + h * a.P + p0 + c) : 0.f;
  }
  if (threadIdx.x < nt) bs[threadIdx.x] = sigmoid_f(ldf<AT>((const AT*)a.beta + (t0 + threadIdx.x) * a.ld_b + h));
  __syncthreads();
  for (int jj = warp; jj < nt; jj += nw) {
    float* dst = kq + jj * 3 * ldn;
    float sk = 0.f, sq = 0.f;
    for (int n = lane; n < N; n += 32) { sk += dst[n] * dst[n]; sq += dst[ldn + n] * dst[ldn + n]; }
    const float ik = 1.f / sqrtf(warp_sum(sk) + a.unit_eps), iq = a.q_scale / sqrtf(warp_sum(sq) + a.unit_eps);
    for (int n = lane; n < N; n += 32) { dst[n] *= ik; dst[ldn + n] *= iq; }
  }
  __syncthreads();
}

// The token-wise part of the delta rule's operands, once per step instead of once per column block, as fp32 rows
// [k unit: G N | q unit * q_scale: G N | decay: H N | v: H P | sigmoid(beta): H] (row stride ld_pre, a multiple of 4 floats), so that
// the scan can fetch them with asynchronous copies.                                                          grid (T), block 256
__host__ __device__ inline long long delta_pre_width(int G, int H, int N, int P) { return ((long long)(2 * G + H) * N + (long long)H * P + H + 3) / 4 * 4; }

template <typename AT>
__global__ void delta_prepare_kernel(DeltaArgs a, float* __restrict__ pre) {
  const long long t = blockIdx.x;
  const int N = a.N, GN = a.G * N, HN = a.H * N, HP = a.H * a.P, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const AT* row = reinterpret_cast<const AT*>(a.in) + t * a.ld_in;
  float* out = pre + t * a.ld_pre;
  for (int gi = warp; gi < a.G; gi += nw) {
    float sk = 0.f, sq = 0.f;
    for (int n = lane; n < N; n += 32) {
      const float qv = ldf<AT>(row + gi * N + n), kv = ldf<AT>(row + GN + gi * N + n);
      sk += kv * kv; sq += qv * qv;
    }
    const float ik = 1.f / sqrtf(warp_sum(sk) + a.unit_eps), iq = a.q_scale / sqrtf(warp_sum(sq) + a.unit_eps);
    for (int n = lane; n < N; n += 32) {
      out[gi * N + n] = ldf<AT>(row + GN + gi * N + n) * ik;
      out[GN + gi * N + n] = ldf<AT>(row + gi * N + n) * iq;
    }
  }
  for (int e = threadIdx.x; e < HN; e += blockDim.x)
    out[2 * GN + e] = expf(-expf(a.A_log[e / N]) * softplus_f(a.dt[t * a.ld_dt + e] + a.dt_bias[e]));
  for (int e = threadIdx.x; e < HP; e += blockDim.x) out[2 * GN + HN + e] = ldf<AT>(row + 2 * GN + e);
  for (int e = threadIdx.x; e < a.H; e += blockDim.x) out[2 * GN + HN + HP + e] = sigmoid_f(ldf<AT>((const AT*)a.beta + t * a.ld_b + e));
}

__device__ __forceinline__ void cp_async_16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

constexpr int kDeltaTokensMax = 16;

// One CTA per (sequence, head, block of PB value columns): the columns of S evolve independently.  S[N][PB] in shared memory; thread
// (r, p) owns rows n = r, r + R, .. of column p.  Per block of tokens the operands are staged by one warp per token (unit vectors of
// q and k by a warp reduction, decays and the write strength in fp32); per token two barriers:
//   S <- g S, partial S^T k  |  u = beta (v - S^T k), S <- S + k u^T, partial S^T q  |  o
template <typename AT>
__global__ void delta_scan_kernel(DeltaArgs a, int PB, int R, int kTok) {
  extern __shared__ __align__(16) float smem[];
  const int b = blockIdx.x, h = blockIdx.y, N = a.N, P = a.P, H = a.H, p0 = blockIdx.z * PB;
  const int g = h / (H / a.G);
  const bool vec4 = PB % 4 == 0 && P % 4 == 0;          // 16-byte copies of the state block (rows of PB floats at a stride of P)
  const int p = threadIdx.x % PB, r = threadIdx.x / PB, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  float* S = smem;                          // [N][PB]
  float* red1 = S + N * PB;                 // [R][PB]
  float* red2 = red1 + R * PB;              // [R][PB]
  float* kq = red2 + R * PB;                // [tokens][3N]   k | q | g
  float* vs = kq + kTok * 3 * N;            // [tokens][PB]
  float* bs = vs + kTok * PB;               // [tokens]
  const int s = a.cu[b], q = a.cu[b + 1] - s;
  if (q == 0) return;
  const bool fresh = a.ctx[b] - q == 0;
  float* gS = a.state + ((long long)a.slots[b] * H + h) * N * P;
  if (vec4) {
    for (int e = 4 * threadIdx.x; e < N * PB; e += 4 * blockDim.x) {
      const int n = e / PB, c = e % PB;
      *reinterpret_cast<float4*>(S + e) = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(gS + n * P + p0 + c);
    }
  } else {
    for (int e = threadIdx.x; e < N * PB; e += blockDim.x) { const int n = e / PB, c = e % PB; S[e] = fresh ? 0.f : gS[n * P + p0 + c]; }
  }
  const AT* in = reinterpret_cast<const AT*>(a.in);
  const float negA = -expf(a.A_log[h]);
  const int GN = a.G * N;
  for (int j0 = 0; j0 < q; j0 += kTok) {
    const int nt = min(kTok, q - j0);
    __syncthreads();                        // the last block's operands are no longer read (and the state is loaded)
    delta_stage<AT>(a, s + j0, nt, h, g, p0, PB, negA, kq, vs, bs, N);
    for (int jj = 0; jj < nt; ++jj) {
      const float* kr = kq + jj * 3 * N;
      if (r < R) {
        float acc = 0.f;
        for (int n = r; n < N; n += R) {
          const float sv = kr[2 * N + n] * S[n * PB + p];
          S[n * PB + p] = sv;
          acc += sv * kr[n];
        }
        red1[r * PB + p] = acc;
      }
      __syncthreads();
      if (r < R) {
        float sk = 0.f;
        for (int i = 0; i < R; ++i) sk += red1[i * PB + p];
        const float u = bs[jj] * (vs[jj * PB + p] - sk);
        float acc = 0.f;
        for (int n = r; n < N; n += R) {
          const float sv = S[n * PB + p] + kr[n] * u;
          S[n * PB + p] = sv;
          acc += sv * kr[N + n];
        }
        red2[r * PB + p] = acc;
      }
      __syncthreads();
      if (r == 0) {
        float y = 0.f;
        for (int i = 0; i < R; ++i) y += red2[i * PB + p];
        a.out[(long long)(s + j0 + jj) * H * P + h * P + p0 + p] = y;
      }
    }
  }
  __syncthreads();
  if (vec4) {
    for (int e = 4 * threadIdx.x; e < N * PB; e += 4 * blockDim.x) {
      const int n = e / PB, c = e % PB;
      *reinterpret_cast<float4*>(gS + n * P + p0 + c) = *reinterpret_cast<const float4*>(S + e);
    }
  } else {
    for (int e = threadIdx.x; e < N * PB; e += blockDim.x) { const int n = e / PB, c = e % PB; gS[n * P + p0 + c] = S[e]; }
  }
}

// The same recurrence with the state in REGISTERS, for portions of many tokens (bound by the latency of a token, not by the state's
// bytes): L lanes share a value column, lane l holding the key rows 4 (l + L j) + e (j < NR4, e < 4: 16-byte shared-memory loads of k, q
// and the decay, consecutive over the lanes), so a warp runs 32 / L columns at once, both products S^T k and S^T q end in log2(L)
// shuffles, and a token needs no block barrier.  The operands of 16 tokens at a time come from delta_prepare_kernel's rows by asynchronous
// copies into one of two buffers while the block before is computed (rows padded with zeros to 4 L NR4, so the token loop has no
// bounds checks).                                                                grid (B, H, ceil(P / PB)), PB = warps * 32 / L
constexpr int kDeltaWarpMinTokens = 8;      // shorter steps are bound by the state copies: the shared-memory kernel with 16-byte copies runs

template <typename AT, int L, int NR4>
__global__ void delta_scan_warp_kernel(DeltaArgs a, int kTok) {
  constexpr int CPW = 32 / L, NP = 4 * L * NR4;
  extern __shared__ __align__(16) float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, PB = nw * CPW;
  const int l = lane % L, cw = lane / L;
  const int b = blockIdx.x, h = blockIdx.y, N = a.N, P = a.P, H = a.H, p0 = blockIdx.z * PB;
  const int g = h / (H / a.G), col = warp * CPW + cw, pc = p0 + col;
  const bool colok = pc < P;
  const int per = 3 * NP + PB + 4;          // floats of one token: k | q | g | v | beta (padded to 16 bytes)
  const int s = a.cu[b], q = a.cu[b + 1] - s;
  if (q == 0) return;
  const bool fresh = a.ctx[b] - q == 0;
  float* gS = a.state + ((long long)a.slots[b] * H + h) * N * P;
  float st[4 * NR4];
#pragma unroll
  for (int j = 0; j < NR4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 4 * (l + L * j) + e;
      st[4 * j + e] = (!fresh && colok && n < N) ? gS[(long long)n * P + pc] : 0.f;
    }
  // both staging buffers start as zeros: rows behind N and columns behind P are never copied
  for (int e = threadIdx.x; e < 2 * kTok * per; e += blockDim.x) smem[e] = 0.f;
  __syncthreads();
  const int GN = a.G * N, HN = H * N, vw = min(PB, P - p0);
  const bool vec = N % 4 == 0 && P % 4 == 0 && PB % 4 == 0;          // 16-byte copies: every segment starts and ends on a 16-byte boundary
  const int n4 = vec ? N / 4 : N, v4 = vec ? vw / 4 : vw, items = 3 * n4 + v4 + 1;
  // asynchronous copies of the operands of tokens t0 .. t0 + nt into buffer `buf`: all of a block are in flight at once
  auto fetch = [&](long long t0, int nt, float* buf) {
    for (int e = threadIdx.x; e < nt * items; e += blockDim.x) {
      const int jj = e / items, c = e - jj * items;
      const float* pr = a.pre + (t0 + jj) * a.ld_pre;
      float* dst = buf + jj * per;
      if (c >= 3 * n4 + v4) { cp_async_4(dst + 3 * NP + PB, pr + 2 * GN + HN + H * P + h); continue; }
      const int seg = c < 3 * n4 ? c / n4 : 3, i = c - seg * n4;
      const float* src = seg == 0 ? pr + g * N : seg == 1 ? pr + GN + g * N : seg == 2 ? pr + 2 * GN + h * N : pr + 2 * GN + HN + h * P + p0;
      float* d = seg == 3 ? dst + 3 * NP : dst + seg * NP;
      if (vec) cp_async_16(d + 4 * i, src + 4 * i); else cp_async_4(d + i, src + i);
    }
    cp_async_commit();
  };
  fetch(s, min(kTok, q), smem);
  int blk = 0;
  for (int j0 = 0; j0 < q; j0 += kTok, ++blk) {
    const int nt = min(kTok, q - j0);
    cp_async_wait_all();
    __syncthreads();                        // this block's operands have landed for every thread; the other buffer is no longer read
    if (j0 + kTok < q) fetch(s + j0 + kTok, min(kTok, q - j0 - kTok), smem + ((blk + 1) & 1) * kTok * per);
    const float* cur = smem + (blk & 1) * kTok * per;
    for (int jj = 0; jj < nt; ++jj) {
      const float* tk = cur + jj * per;
      const float4* k4 = reinterpret_cast<const float4*>(tk) + l;
      const float4* q4 = k4 + NP / 4;
      const float4* g4 = k4 + 2 * (NP / 4);
      float a0 = 0.f, a1 = 0.f;
#pragma unroll
      for (int j = 0; j < NR4; ++j) {
        const float4 kk = k4[j * L], gg = g4[j * L];
        st[4 * j] *= gg.x; st[4 * j + 1] *= gg.y; st[4 * j + 2] *= gg.z; st[4 * j + 3] *= gg.w;
        a0 += st[4 * j] * kk.x + st[4 * j + 2] * kk.z;
        a1 += st[4 * j + 1] * kk.y + st[4 * j + 3] * kk.w;
      }
      float sk = a0 + a1;
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) sk += __shfl_xor_sync(0xffffffffu, sk, o);
      const float u = tk[3 * NP + PB] * (tk[3 * NP + col] - sk);
      a0 = 0.f; a1 = 0.f;
#pragma unroll
      for (int j = 0; j < NR4; ++j) {
        const float4 kk = k4[j * L], qq = q4[j * L];
        st[4 * j] += kk.x * u; st[4 * j + 1] += kk.y * u; st[4 * j + 2] += kk.z * u; st[4 * j + 3] += kk.w * u;
        a0 += st[4 * j] * qq.x + st[4 * j + 2] * qq.z;
        a1 += st[4 * j + 1] * qq.y + st[4 * j + 3] * qq.w;
      }
      float y = a0 + a1;
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (l == 0 && colok) a.out[(long long)(s + j0 + jj) * H * P + h * P + pc] = y;
    }
  }
#pragma unroll
  for (int j = 0; j < NR4; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = 4 * (l + L * j) + e;
      if (colok && n < N) gS[(long long)n * P + pc] = st[4 * j + e];
    }
}

// ---------------------------------------------------------------------------------------------------------- minGRU
// z = sigmoid(rows[z]), c = u + 1/2 (u >= 0) or sigmoid(u), S <- (1 - z) S + z c, out = S * silu(rows[g]) * out_mult.
// The recurrence is linear in S, so a sequence's tokens are cut into TS slices: thread (channel, slice) first folds its slice into
// (A, B) with S_end = A S_start + B, then takes its start from the slices before it (at most TS - 1 steps) and runs its slice again,
// writing the outputs.  Decode (one token) is the TS = 1 case.                     grid (B, ceil(R / 32)), block (32 channels, TS)
template <typename AT>
__global__ void mingru_scan_kernel(const AT* __restrict__ rows, long long ld, int z0, int x0, int g0, int R, float* __restrict__ state,
                                   const int* __restrict__ cu, const int* __restrict__ ctx, const int* __restrict__ slots, float out_mult,
                                   AT* __restrict__ out, long long ld_out) {
  __shared__ float fa[32][33], fb[32][33];
  const int b = blockIdx.x, cl = threadIdx.x, sl = threadIdx.y, TS = blockDim.y, c = blockIdx.y * 32 + cl;
  const int s = cu[b], q = cu[b + 1] - s;
  if (q == 0) return;
  const int len = (q + TS - 1) / TS, j0 = min(q, sl * len), j1 = min(q, j0 + len);
  const bool live = c < R;
  const AT* row = rows + (long long)(s + j0) * ld + c;
  float A = 1.f, Bv = 0.f;
  if (live && TS > 1) {
    const AT* r = row;
#pragma unroll 4
    for (int j = j0; j < j1; ++j, r += ld) {
      const float z = sigmoid_f(ldf<AT>(r + z0)), u = ldf<AT>(r + x0);
      const float cand = u >= 0.f ? u + 0.5f : sigmoid_f(u);
      A *= 1.f - z;
      Bv = (1.f - z) * Bv + z * cand;
    }
  }
  fa[sl][cl] = A; fb[sl][cl] = Bv;
  __syncthreads();
  if (!live) return;
  float* st = state + (long long)slots[b] * R + c;
  float S = ctx[b] - q == 0 ? 0.f : *st;
  for (int i = 0; i < sl; ++i) S = fa[i][cl] * S + fb[i][cl];
  AT* orow = out + (long long)(s + j0) * ld_out + c;
#pragma unroll 4
  for (int j = j0; j < j1; ++j, row += ld, orow += ld_out) {
    const float z = sigmoid_f(ldf<AT>(row + z0)), u = ldf<AT>(row + x0), gr = ldf<AT>(row + g0);
    const float cand = u >= 0.f ? u + 0.5f : sigmoid_f(u);
    S = (1.f - z) * S + z * cand;
    stf<AT>(orow, S * silu_f(gr) * out_mult);
  }
  if (sl == TS - 1) *st = S;          // the last slice ends at the sequence's last token (empty slices pass S through)
}

// ---------------------------------------------------------------------------------------------------------- attention prologue
struct PrologueArgs {
  const void* rows; long long ld;           // AT, query heads from column q0 on, keys k0, values v0
  int q0, k0, v0, H, G, D, V;
  const float* qn; const float* kn;         // [D] norm weights, [H D] / [G D] with `whole` (nullable)
  bool whole;                               // ONE norm over all query (key) heads' entries instead of one per head (before the rotation only)
  float eps;
  const float* inv_freq; int rot;           // angles per position of the rot / 2 pairs
  float rot_mult;                           // factor on cos and sin
  const int* positions; const int* slot_map;
  int page;
  const void* v_first; long long ld_vf;     // AT [T, G V] mixed into the values (nullable)
  float lam;
  float* qout; void* kpool; void* vpool;
};

// One warp per head of a token (query heads first, then key heads), the head's entries lane + 32 i in registers: RMS norm (times a weight)
// and rotation of the first `rot` entries, adjacent pairs (2i, 2i+1) or HALF pairs (i, i + rot / 2), the norm before the rotation or
// (AFTER) behind it.  The token's cosines and sines are computed once per CTA.  Queries -> qout fp32 [T, H, D]; keys and values (as they
// are, or (1 - lam) v + lam v_first) -> the paged pools.
template <typename AT, int NPL, bool HALF, bool AFTER>
__global__ void qk_norm_rope_append_kernel(PrologueArgs a) {
  extern __shared__ float cs[];             // [rot / 2] cosines | [rot / 2] sines
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, D = a.D, H = a.H, G = a.G, V = a.V, hr = a.rot / 2;
  const float pos = (float)a.positions[t];
  for (int i = threadIdx.x; i < hr; i += blockDim.x) {
    float sn, cn;
    sincosf(pos * a.inv_freq[i], &sn, &cn);
    cs[i] = cn * a.rot_mult; cs[hr + i] = sn * a.rot_mult;
  }
  __syncthreads();
  const int slot = a.slot_map[t], pg = slot / a.page, off = slot % a.page;
  const AT* r = (const AT*)a.rows + t * a.ld;
  float inv_q = 1.f, inv_k = 1.f;
  if (a.whole) {
    __shared__ float red[32];
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < H * D; i += blockDim.x) { const float v = ldf<AT>(r + a.q0 + i); sq += v * v; }
    for (int i = threadIdx.x; i < G * D; i += blockDim.x) { const float v = ldf<AT>(r + a.k0 + i); sk += v * v; }
    inv_q = 1.f / sqrtf(block_sum(sq, red) / (float)(H * D) + a.eps);
    inv_k = 1.f / sqrtf(block_sum(sk, red) / (float)(G * D) + a.eps);
  }
  for (int hh = warp; hh < H + G; hh += nw) {
    const bool isq = hh < H;
    const AT* src = isq ? r + a.q0 + hh * D : r + a.k0 + (hh - H) * D;
    const float* w = isq ? a.qn : a.kn;
    if (a.whole && w != nullptr) w += (isq ? hh : hh - H) * D;
    float v[NPL], inv = 1.f;
#pragma unroll
    for (int i = 0; i < NPL; ++i) v[i] = lane + 32 * i < D ? ldf<AT>(src + lane + 32 * i) : 0.f;
    auto scale = [&]() {
      if (a.whole) {
        inv = isq ? inv_q : inv_k;
      } else {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NPL; ++i) ss += v[i] * v[i];
        inv = 1.f / sqrtf(warp_sum(ss) / (float)D + a.eps);
      }
#pragma unroll
      for (int i = 0; i < NPL; ++i) { const int d = lane + 32 * i; v[i] *= w != nullptr && d < D ? inv * w[d] : inv; }
    };
    if (!AFTER) scale();
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      const int d = lane + 32 * i;
      if (32 * i >= a.rot) break;             // uniform over the warp: all lanes take part in the shuffle
      if (HALF) {
        if (d < a.rot) {
          const bool lo = d < hr;
          const int p = lo ? d + hr : d - hr, k = lo ? d : p;
          float other = ldf<AT>(src + p);
          if (!AFTER) other *= w != nullptr ? inv * w[p] : inv;
          v[i] = lo ? v[i] * cs[k] - other * cs[hr + k] : v[i] * cs[k] + other * cs[hr + k];
        }
      } else {
        const float other = __shfl_xor_sync(0xffffffffu, v[i], 1);      // d even <-> lane even
        if (d < a.rot) v[i] = (d & 1) ? v[i] * cs[d >> 1] + other * cs[hr + (d >> 1)] : v[i] * cs[d >> 1] - other * cs[hr + (d >> 1)];
      }
    }
    if (AFTER) scale();
    float* qd = a.qout + (t * H + hh) * D;
    AT* kd = (AT*)a.kpool + (((long long)pg * G + (hh - H)) * a.page + off) * D;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      const int d = lane + 32 * i;
      if (d < D) { if (isq) qd[d] = v[i]; else stf<AT>(kd + d, v[i]); }
    }
  }
  AT* vpool = (AT*)a.vpool;
  const AT* vf = a.v_first != nullptr ? (const AT*)a.v_first + t * a.ld_vf : nullptr;
  for (int i = threadIdx.x; i < G * V; i += blockDim.x) {
    AT* dst = vpool + (((long long)pg * G + i / V) * a.page + off) * V + i % V;
    if (vf == nullptr) *dst = r[a.v0 + i];
    else stf<AT>(dst, (1.f - a.lam) * ldf<AT>(r + a.v0 + i) + a.lam * ldf<AT>(vf + i));
  }
}

// The form without rotation, value mixing and heads to tell apart: one norm over the query row and one over the key row, four entries per
// thread and step, the row in registers (NQ steps of 256 threads; sizes multiples of 4, rows and pools aligned to four entries).
template <typename AT, int NQ>
__global__ void __launch_bounds__(256) whole_norm_append_kernel(PrologueArgs a) {
  __shared__ float red[2][8];
  const long long t = blockIdx.x;
  const int D = a.D, V = a.V, G = a.G, nq = a.H * D / 4, nk = G * D / 4, nv = G * V / 4;
  const AT* r = (const AT*)a.rows + t * a.ld;
  float q[NQ][4], k[NQ][4], sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int c = threadIdx.x + 256 * i;
    if (c < nq) load4<AT>(r + a.q0 + 4 * c, q[i]);
    if (c < nk) load4<AT>(r + a.k0 + 4 * c, k[i]);
  }
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int c = threadIdx.x + 256 * i;
#pragma unroll
    for (int e = 0; e < 4; ++e) { if (c < nq) sq += q[i][e] * q[i][e]; if (c < nk) sk += k[i][e] * k[i][e]; }
  }
  sq = warp_sum(sq); sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
  const int slot = a.slot_map[t], pg = slot / a.page, off = slot % a.page;
  for (int c = threadIdx.x; c < nv; c += 256) {
    const int h = 4 * c / V, d = 4 * c - h * V;
    float f[4];
    load4<AT>(r + a.v0 + 4 * c, f);
    store4<AT>((AT*)a.vpool + (((long long)pg * G + h) * a.page + off) * V + d, f);
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) { sq += red[0][w]; sk += red[1][w]; }
  const float iq = 1.f / sqrtf(sq / (float)(4 * nq) + a.eps), ik = 1.f / sqrtf(sk / (float)(4 * nk) + a.eps);
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int c = threadIdx.x + 256 * i;
    float w[4] = {1.f, 1.f, 1.f, 1.f};
    if (c < nq) {
      if (a.qn != nullptr) load4<float>(a.qn + 4 * c, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) q[i][e] *= iq * w[e];
      store4<float>(a.qout + 4 * (t * nq + c), q[i]);
    }
    if (c < nk) {
      if (a.kn != nullptr) load4<float>(a.kn + 4 * c, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) k[i][e] *= ik * w[e];
      const int h = 4 * c / D, d = 4 * c - h * D;
      store4<AT>((AT*)a.kpool + (((long long)pg * G + h) * a.page + off) * D + d, k[i]);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------- router
// One warp per token.  s = softmax(z) over all E experts; choice c = s + corr; groups = ng equal runs of neighbours, a group's value is
// its largest c; experts outside the `keep` best groups count as -inf; the `top` largest c win (ties: lowest id); weights = their s.
__global__ void group_softmax_topk_kernel(const float* __restrict__ z, long long ld_z, const float* __restrict__ corr, int E, int top, int ng, int keep,
                                          int* __restrict__ idx, float* __restrict__ w) {
  extern __shared__ float sh[];
  float* sc = sh;                            // [E] plain scores
  float* ch = sh + E;                        // [E] choice scores
  float* gv = ch + E;                        // [ng]
  const long long t = blockIdx.x;
  const int lane = threadIdx.x;
  float mx = -INFINITY;
  for (int e = lane; e < E; e += 32) mx = fmaxf(mx, z[t * ld_z + e]);
  mx = warp_max(mx);
  float sum = 0.f;
  for (int e = lane; e < E; e += 32) { const float v = expf(z[t * ld_z + e] - mx); sc[e] = v; sum += v; }
  sum = warp_sum(sum);
  for (int e = lane; e < E; e += 32) { const float s = sc[e] / sum; sc[e] = s; ch[e] = s + (corr != nullptr ? corr[e] : 0.f); }
  __syncwarp();
  if (ng > 1 && keep < ng) {
    const int per = E / ng;
    for (int gi = lane; gi < ng; gi += 32) {
      float b = -INFINITY;
      for (int e = gi * per; e < (gi + 1) * per; ++e) b = fmaxf(b, ch[e]);
      gv[gi] = b;
    }
    __syncwarp();
    // drop the ng - keep worst groups: repeatedly the smallest value, ties to the HIGHEST id (so that kept ties go to the lowest)
    for (int j = 0; j < ng - keep; ++j) {
      float worst = INFINITY; int wi = -1;
      for (int gi = lane; gi < ng; gi += 32) { const float v = gv[gi]; if (v <= worst) { worst = v; wi = gi; } }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, worst, o);
        const int oi = __shfl_xor_sync(0xffffffffu, wi, o);
        if (oi >= 0 && (wi < 0 || ov < worst || (ov == worst && oi > wi))) { worst = ov; wi = oi; }
      }
      if (lane == 0) gv[wi] = INFINITY;      // marked as dropped
      __syncwarp();
      for (int e = wi * per + lane; e < (wi + 1) * per; e += 32) ch[e] = -INFINITY;
      __syncwarp();
    }
  }
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY; int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) { const float v = ch[e]; if (v > best) { best = v; bi = e; } }   // ascending e: first maximum wins
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if (lane == 0) { idx[t * top + j] = bi; w[t * top + j] = sc[bi]; ch[bi] = -INFINITY; }
    __syncwarp();
  }
}

}  // namespace

// =========================================================================================================== launchers
cudaError_t stream_embed_launch(const void* table, bool table_f32, long long ld, const long long* ids, float scale, int S, int n, float* xs, const void* pos,
                                const int* positions, int n_pos, int T, cudaStream_t s) {
  if (S < 1 || S > kMaxStreams) return cudaErrorInvalidValue;
  dim3 grid(T, (n + 1023) / 1024);
  AT_DISPATCH(table_f32, (stream_embed_kernel<AT><<<grid, 256, 0, s>>>((const AT*)table, ld, ids, scale, S, n, xs, (const AT*)pos, positions, n_pos)));
  return last();
}

cudaError_t hyper_step_launch(float* xs, const float* y, long long ld_y, const float* y2, long long ld_y2, const void* gate, long long ld_g,
                              const float* ls, const float* mix, const float* out_w, float mult, const float* in_w, float alpha, const float* w,
                              const float* b, void* xa, bool f32, int S, int n, int T, cudaStream_t s) {
  if (S < 1 || S > kMaxStreams) return cudaErrorInvalidValue;
  HyperArgs a{xs, y, ld_y, y2, ld_y2, gate, ld_g, ls, mix, out_w, in_w, w, b, mult, alpha, xa, S, n};
  dim3 grid(T, (n + 255) / 256);
  AT_DISPATCH(f32, (hyper_step_kernel<AT><<<grid, 256, 0, s>>>(a)));
  return last();
}

cudaError_t relu2_launch(void* x, long long ld, int n, bool f32, int T, cudaStream_t s) {
  dim3 grid(T, (n + 1023) / 1024);
  AT_DISPATCH(f32, (relu2_kernel<AT><<<grid, 256, 0, s>>>((AT*)x, ld, n)));
  return last();
}

cudaError_t delta_scan_launch(const void* in, long long ld_in, const void* beta, long long ld_b, const float* dt, long long ld_dt,
                              const float* dt_bias, const float* A_log, float* state, const int* cu, const int* ctx, const int* slots, float* out,
                              int B, int H, int G, int N, int P, float q_scale, float unit_eps, bool f32, int max_q, float* pre, int T, cudaStream_t s) {
  if (G < 1 || H % G != 0 || P < 1 || N < 1) return cudaErrorInvalidValue;
  DeltaArgs a{in, ld_in, beta, ld_b, dt, ld_dt, dt_bias, A_log, state, cu, ctx, slots, out, H, G, N, P, q_scale, unit_eps, nullptr, 0};
  if (delta_scan_wants_prepare(N, max_q)) {
    if (pre == nullptr) return cudaErrorInvalidValue;
    a.pre = pre; a.ld_pre = delta_pre_width(G, H, N, P);
    AT_DISPATCH(f32, (delta_prepare_kernel<AT><<<T, 256, 0, s>>>(a, pre)));
    // register form: 4 lanes per value column (8 beyond 128 key rows), up to 4 warps per CTA.  A warp's time per token is its serial
    // instruction count, so while the grid leaves SMs idle (one short batch) a column is spread over more lanes: fewer rows per lane,
    // one more shuffle level, twice the CTAs
    int L = N <= 128 ? 4 : 8;
    auto ctas = [&](int lanes) { const int pb = 4 * (32 / lanes); return (long long)B * H * ((P + pb - 1) / pb); };
    while (L < 16 && ctas(L) < 148 && N > 4 * L) L *= 2;
    const int cpw = 32 / L;
    const int need = (N + 4 * L - 1) / (4 * L), nr4 = need <= 1 ? 1 : need <= 2 ? 2 : need <= 4 ? 4 : 8;
    int nwarps = (P + cpw - 1) / cpw;
    if (nwarps > 4) nwarps = 4;
    const int PB = nwarps * cpw, NP = 4 * L * nr4;
    const int stage = max_q < kDeltaTokensMax ? max_q : kDeltaTokensMax;
    const size_t smem = 2 * (size_t)stage * (3 * NP + PB + 4) * sizeof(float);
    auto go = [&](auto k) -> cudaError_t {
      if (smem > 48 * 1024) { cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); if (e != cudaSuccess) return e; }
      k<<<dim3(B, H, (P + PB - 1) / PB), 32 * nwarps, smem, s>>>(a, stage);
      return last();
    };
#define DELTA_CASE(LL, R) if (L == LL && nr4 == R) { AT_DISPATCH(f32, return go(delta_scan_warp_kernel<AT, LL, R>)); }
    DELTA_CASE(4, 1) DELTA_CASE(4, 2) DELTA_CASE(4, 4) DELTA_CASE(4, 8)
    DELTA_CASE(8, 1) DELTA_CASE(8, 2) DELTA_CASE(8, 4) DELTA_CASE(8, 8)
    DELTA_CASE(16, 1) DELTA_CASE(16, 2) DELTA_CASE(16, 4)
#undef DELTA_CASE
    return cudaErrorInvalidValue;
  }
  // columns of the state are independent: split a head's value dimension over CTAs (PB columns each) while the grid is small
  int PB = P;
  while (PB > 16 && PB % 2 == 0 && ((long long)B * H * (P / PB) < 592 || PB > 256)) PB /= 2;
  if (PB > 1024) return cudaErrorInvalidValue;
  int R = 256 / PB;
  if (R < 1) R = 1;
  if (R > N) R = N;
  const int threads = (R * PB + 31) / 32 * 32;   // tail threads (r >= R) only help with staging and the state copy
  int stage = max_q < 1 ? 1 : (max_q < kDeltaTokensMax ? max_q : kDeltaTokensMax);
  auto bytes = [&](int st) { return ((size_t)N * PB + 2 * (size_t)R * PB + (size_t)st * (3 * N + PB + 1)) * sizeof(float); };
  while (stage > 1 && bytes(stage) > 200 * 1024) stage /= 2;
  const size_t smem = bytes(stage);
  if (smem > 220 * 1024) return cudaErrorInvalidValue;
  if (f32) {
    auto k = delta_scan_kernel<float>;
    if (smem > 48 * 1024) { cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); if (e != cudaSuccess) return e; }
    k<<<dim3(B, H, P / PB), threads, smem, s>>>(a, PB, R, stage);
  } else {
    auto k = delta_scan_kernel<__nv_bfloat16>;
    if (smem > 48 * 1024) { cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); if (e != cudaSuccess) return e; }
    k<<<dim3(B, H, P / PB), threads, smem, s>>>(a, PB, R, stage);
  }
  return last();
}

cudaError_t mingru_scan_launch(const void* rows, long long ld, int z0, int x0, int g0, int R, float* state, const int* cu, const int* ctx,
                               const int* slots, float out_mult, void* out, long long ld_out, int B, bool f32, int max_q, cudaStream_t s) {
  int TS = 1;                                   // slices of at least 16 tokens, at most 32 of them
  while (TS < 32 && max_q >= 32 * TS) TS *= 2;
  dim3 grid(B, (R + 31) / 32), block(32, TS);
  AT_DISPATCH(f32, (mingru_scan_kernel<AT><<<grid, block, 0, s>>>((const AT*)rows, ld, z0, x0, g0, R, state, cu, ctx, slots, out_mult, (AT*)out, ld_out)));
  return last();
}

template <typename AT, int NPL>
static void prologue_t(const PrologueArgs& a, bool half, bool after, int T, cudaStream_t s) {
  const int threads = 32 * (a.H + a.G < 8 ? a.H + a.G : 8);
  const size_t smem = (a.rot < 2 ? 2 : a.rot) * sizeof(float);
  if (half) {
    if (after) qk_norm_rope_append_kernel<AT, NPL, true, true><<<T, threads, smem, s>>>(a);
    else qk_norm_rope_append_kernel<AT, NPL, true, false><<<T, threads, smem, s>>>(a);
  } else {
    if (after) qk_norm_rope_append_kernel<AT, NPL, false, true><<<T, threads, smem, s>>>(a);
    else qk_norm_rope_append_kernel<AT, NPL, false, false><<<T, threads, smem, s>>>(a);
  }
}

cudaError_t qk_norm_rope_append_launch(const void* rows, long long ld, int q0, int k0, int v0, int H, int G, int D, int V, const float* qn,
                                       const float* kn, float eps, const float* inv_freq, int rot, const int* positions, const int* slot_map,
                                       int page, float* qout, void* kpool, void* vpool, bool f32, bool half, bool norm_after, float rot_mult,
                                       const void* v_first, long long ld_vf, float lam, bool whole, int T, cudaStream_t s) {
  if (rot % 2 != 0 || rot > D || D > 1024 || (whole && norm_after)) return cudaErrorInvalidValue;
  const PrologueArgs a{rows, ld, q0, k0, v0, H, G, D, V, qn, kn, whole, eps, inv_freq, rot, rot_mult, positions, slot_map, page, v_first, ld_vf, lam, qout, kpool, vpool};
  const int n4 = H * D / 4, es = f32 ? 4 : 2;
  auto al = [](const void* p, int b) { return reinterpret_cast<uintptr_t>(p) % b == 0; };
  if (whole && rot == 0 && v_first == nullptr && G <= H && D % 4 == 0 && V % 4 == 0 && ld % 4 == 0 && q0 % 4 == 0 && k0 % 4 == 0 && v0 % 4 == 0 && n4 <= 8 * 256 &&
      al(rows, 4 * es) && al(kpool, 4 * es) && al(vpool, 4 * es) && al(qn, 16) && al(kn, 16) && al(qout, 16)) {
    if (n4 <= 256) AT_DISPATCH(f32, (whole_norm_append_kernel<AT, 1><<<T, 256, 0, s>>>(a)));
    else if (n4 <= 2 * 256) AT_DISPATCH(f32, (whole_norm_append_kernel<AT, 2><<<T, 256, 0, s>>>(a)));
    else if (n4 <= 4 * 256) AT_DISPATCH(f32, (whole_norm_append_kernel<AT, 4><<<T, 256, 0, s>>>(a)));
    else AT_DISPATCH(f32, (whole_norm_append_kernel<AT, 8><<<T, 256, 0, s>>>(a)));
    return last();
  }
  if (D <= 64) AT_DISPATCH(f32, (prologue_t<AT, 2>(a, half, norm_after, T, s)));
  else if (D <= 128) AT_DISPATCH(f32, (prologue_t<AT, 4>(a, half, norm_after, T, s)));
  else if (D <= 256) AT_DISPATCH(f32, (prologue_t<AT, 8>(a, half, norm_after, T, s)));
  else AT_DISPATCH(f32, (prologue_t<AT, 32>(a, half, norm_after, T, s)));
  return last();
}

bool delta_scan_wants_prepare(int N, int max_q) { return N <= 256 && max_q >= kDeltaWarpMinTokens; }
long long delta_scan_prepare_width(int G, int H, int N, int P) { return delta_pre_width(G, H, N, P); }

cudaError_t group_softmax_topk_launch(const float* z, long long ld_z, const float* corr, int E, int top, int ng, int keep, int* idx, float* w, int T,
                                      cudaStream_t s) {
  if (top > E || ng < 1 || E % ng != 0 || keep < 1 || keep > ng || (size_t)(2 * E + ng) * sizeof(float) > 48 * 1024) return cudaErrorInvalidValue;
  group_softmax_topk_kernel<<<T, 32, (2 * E + ng) * sizeof(float), s>>>(z, ld_z, corr, E, top, ng, keep, idx, w);
  return last();
}
}  // namespace b200
