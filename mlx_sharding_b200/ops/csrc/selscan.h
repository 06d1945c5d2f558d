// Host launch API of selscan.cu (selective scan with one step size per channel).  `f32` selects the activation type of the call: float
// (exact mode) or bf16 (serving); step sizes, decays, recurrence constants and the state are always float.
#pragma once
#include <cuda_runtime.h>

namespace b200 {
// time slices of a step (1: no workspace) and floats of workspace for it
int selective_scan_slices(int B, int I, int N, int max_q);
long long selective_scan_workspace(int B, int I, int N, int slices);
bool selective_scan_supported(int N);
// gate nullable; ws: selective_scan_workspace floats when slices > 1
cudaError_t selective_scan_launch(const void* x, long long ld_x, const float* dt, long long ld_dt, const float* dt_bias, const float* A_log, const void* bc,
                                  long long ld_bc, int b0, int c0, const float* D, const void* gate, long long ld_g, float* state, const int* cu,
                                  const int* ctx, const int* slots, void* out, int B, int I, int N, bool f32, int max_q, int slices, float* ws,
                                  cudaStream_t s);
}  // namespace b200
