// Internal interface of the projections of the layer-list models (dense.cu, dense_tc.cu).
#pragma once
#include "stream.cuh"

struct DenseCall {
  int dtype;             // JG_F32 / JG_BF16
  int epilogue;          // JG_DENSE_*
  int M, N, K;
  const void* x;         // T [M][ldx], or null: rows come from the residual stream through `st`
  int ldx;
  StreamArgs st;
  const void* w[3];      // T [N][ldw], zero between K and ldw
  int ldw;
  const float* bias[3];  // fp32 [N] or null
  void* y;               // T or (out_f32) float [M][ldy]
  int ldy, out_f32;
  float limit;                        // GLU
  float* state;                       // MINGRU: [slots][N]
  const int32_t *pos, *seq;           // MINGRU: [M]
  unsigned long long* key;            // LOGITS: [M]
};
int jg_dense_call(jg_dev* dev, const DenseCall& c);
// bf16, any row count, tcgen05 (epilogues STORE and GLU)
int jg_dense_tc(jg_dev* dev, const DenseCall& c);
