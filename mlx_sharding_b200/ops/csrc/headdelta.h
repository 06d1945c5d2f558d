// Host launch API of headdelta.cu (gated delta rule with one decay per head).  `f32` selects the activation type of the call: float (exact
// mode) or bf16 (serving); unit vectors, decays, write strengths and the state are always float.
#pragma once
#include <cuda_runtime.h>

namespace b200 {
struct HeadDeltaArgs {
  const void* in; long long ld_in;          // activation type: [q: G N | k: G N | v: H P] (after the short convolution)
  const void* beta; long long ld_b;         // raw write strengths, activation type [T, >= H]
  const void* dt; long long ld_dt;          // raw step sizes, activation type [T, >= H]
  const float* dt_bias; const float* A_log; // [H]
  float* state;                             // [slots, H, N, P]
  const int* cu; const int* ctx; const int* slots;
  float* out;                               // fp32 [T, H P]
  int B, T, H, G, N, P;
  float q_scale, unit_eps;
  float* pre;                               // head_delta_workspace floats (portions), unused by steps of single tokens
  int NP;                                   // row width of the workspace (set by the launcher)
};
bool head_delta_supported(int N);
// floats of workspace of a step whose longest portion has max_q tokens (0: none)
long long head_delta_workspace(const HeadDeltaArgs& a, int max_q);
cudaError_t head_delta_launch(HeadDeltaArgs a, bool f32, int max_q, cudaStream_t s);
}  // namespace b200
