// Host launch API of sinkattn.cu (grouped-query attention over paged keys / values with a sink in the softmax, inside blocks of positions
// or a sliding window beside kept first tokens, with a gate per head) and of the tensor-core form of it in attention_prefill.cu.
#pragma once
#include <cuda_runtime.h>

namespace b200 {
struct SinkAttnArgs {
  const float* q;                           // fp32 [T, H, D] (normed, rotated)
  const void* kpool; const void* vpool;     // [pages, G, page, D] / [pages, G, page, V] in the activation type
  const float* sink;                        // [H] (nullable)
  const int* block_tables; int max_blocks;
  const int* positions; const int* cu; int B;
  int H, G, D, V, page;
  int page_shift;                           // log2(page), -1 when page is no power of two
  // visible keys j <= p: same block of `block` positions (0: all) and p - j < window (0: all), or j < keep
  int block, window, keep;
  float scale, out_mult;
  // what is added to the score of a key n = p - j tokens back: -slopes[h] n and bias[h * bias_len + min(n, bias_len - 1)] (both nullable)
  const float* slopes; const float* bias; int bias_len;
  const void* gate; long long ld_gate;      // activation type: the result times sigmoid(gate) (nullable); one logit per head [T, H] or,
  bool gate_elem;                           // with gate_elem, per element [T, H V]
  void* out; long long ld_out;              // activation type, row t at out + t * ld_out, head h at column h * V
  int nsplit, chunk;                        // keys split into nsplit parts of `chunk` visible keys
  int bias_keys;                            // most visible keys of a CTA when their biases are kept in shared memory (0: evaluated key by key)
  float* part;                              // [T, H, nsplit, V + 2] = (m, l, o[V]) when nsplit > 1
};
// query heads one CTA serves for these sizes
int sink_attention_heads_per_cta(int H, int G, int D, int V);
// granularity of `chunk`
int sink_attention_chunk_unit();
// keys of a CTA whose biases shared memory takes
int sink_attention_bias_keys();
cudaError_t sink_attention_launch(const SinkAttnArgs& a, bool f32, int T, cudaStream_t s);
// bf16 on the tensor cores, 64 query rows per CTA (context_lens instead of positions; nsplit, chunk, part unused)
bool sink_flash_supported(int D, int V);
int sink_flash_bias_max();                  // longest distance table (slopes and a table together: the vector form alone)
cudaError_t sink_flash_launch(const SinkAttnArgs& a, const int* context_lens, int max_tiles, cudaStream_t s);
}  // namespace b200
