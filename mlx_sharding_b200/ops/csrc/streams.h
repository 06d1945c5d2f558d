// Host launch API of streams.cu (several residual streams with dynamic-tanh norms, gated delta rule, attention prologue, minGRU,
// group-limited softmax router).  `f32` selects the activation type of the call: float (exact mode) or
// bf16 (serving); streams, norm weights, recurrence constants and states are always float.  Nullable pointers are marked.
#pragma once
#include <cuda_runtime.h>

namespace b200 {
// pos [n_pos, n] in the table's type, added at positions[t] (nullable)
cudaError_t stream_embed_launch(const void* table, bool table_f32, long long ld, const long long* ids, float scale, int S, int n, float* xs, const void* pos,
                                const int* positions, int n_pos, int T, cudaStream_t s);
// y == nullptr: only the read.  y2, gate, ls nullable.
cudaError_t hyper_step_launch(float* xs, const float* y, long long ld_y, const float* y2, long long ld_y2, const void* gate, long long ld_g,
                              const float* ls, const float* mix, const float* out_w, float mult, const float* in_w, float alpha, const float* w,
                              const float* b, void* xa, bool f32, int S, int n, int T, cudaStream_t s);
cudaError_t relu2_launch(void* x, long long ld, int n, bool f32, int T, cudaStream_t s);
cudaError_t delta_scan_launch(const void* in, long long ld_in, const void* beta, long long ld_b, const float* dt, long long ld_dt,
                              const float* dt_bias, const float* A_log, float* state, const int* cu, const int* ctx, const int* slots, float* out,
                              int B, int H, int G, int N, int P, float q_scale, float unit_eps, bool f32, int max_q, float* pre, int T, cudaStream_t s);
// true: the step runs the register form of the scan, which takes a workspace `pre` of T * delta_scan_prepare_width(..) floats (token-wise
// operands, computed once per step)
bool delta_scan_wants_prepare(int N, int max_q);
long long delta_scan_prepare_width(int G, int H, int N, int P);
cudaError_t mingru_scan_launch(const void* rows, long long ld, int z0, int x0, int g0, int R, float* state, const int* cu, const int* ctx,
                               const int* slots, float out_mult, void* out, long long ld_out, int B, bool f32, int max_q, cudaStream_t s);
// qn, kn, v_first nullable; whole: one norm over all query (key) heads' entries, weights [H D] / [G D]
cudaError_t qk_norm_rope_append_launch(const void* rows, long long ld, int q0, int k0, int v0, int H, int G, int D, int V, const float* qn,
                                       const float* kn, float eps, const float* inv_freq, int rot, const int* positions, const int* slot_map,
                                       int page, float* qout, void* kpool, void* vpool, bool f32, bool half, bool norm_after, float rot_mult,
                                       const void* v_first, long long ld_vf, float lam, bool whole, int T, cudaStream_t s);
cudaError_t group_softmax_topk_launch(const float* z, long long ld_z, const float* corr, int E, int top, int ng, int keep, int* idx, float* w, int T,
                                      cudaStream_t s);
}  // namespace b200
