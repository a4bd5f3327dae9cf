// Internal interface of the projections of the layer-list models (dense.cu, dense_tc.cu).
#pragma once
#include "stream.cuh"

// What STORE does beyond the bias: an activation on columns [lo, hi), and columns from `split` on in fp32 elsewhere.
struct DenseOut {
  int act = JG_ACT_NONE, lo = 0, hi = 0, split = 1 << 30, ld2 = 0, ld_side = 0, col_side = 0, vocab = 0;
  float* y2 = nullptr;
  const void* side = nullptr;  // T [vocab][ld_side]
  const int32_t* tokens = nullptr;
};
#ifdef __CUDACC__
// what the row's token has in the table for a column; an id outside the table reads as zero (from row 0, so that no branch
// keeps several of these loads apart)
template <typename T>
__device__ __forceinline__ const T* dense_side_ptr(const DenseOut& o, int tok, int col) {
  return reinterpret_cast<const T*>(o.side) + (size_t)(tok >= 0 && tok < o.vocab ? tok : 0) * o.ld_side + o.col_side + col;
}
template <typename T>
__device__ __forceinline__ float dense_side(const DenseOut& o, int row, int col) {
  if (o.act != JG_ACT_GELU_SIDE) return 0.f;
  const int tok = o.tokens[row];
  const float v = to_f32(*dense_side_ptr<T>(o, tok, col));
  return tok >= 0 && tok < o.vocab ? v : 0.f;
}
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }
// side: dense_side of the same row and column, which the caller may have loaded ahead
__device__ __forceinline__ float dense_act(const DenseOut& o, int col, float v, float side) {
  if (o.act == JG_ACT_NONE || col < o.lo || col >= o.hi) return v;
  if (o.act == JG_ACT_SILU) return silu_f32(v);
  if (o.act == JG_ACT_RELU2) { v = fmaxf(v, 0.f); return v * v; }
  return gelu_tanh_f32(v) * side;
}
#endif

struct DenseCall {
  int dtype;             // JG_F32 / JG_BF16
  int epilogue;          // JG_DENSE_*
  int M, N, K;
  const void* x;         // T [M][ldx], or null: rows come from the residual stream through `st`
  int ldx;
  StreamArgs st;
  const jg_gated_desc* gated;  // or null; columns from `lead` on (1-2 rows)
  int lead;
  const void* w[3];      // T [N][ldw], zero between K and ldw
  int ldw;
  const float* bias[3];  // fp32 [N] or null
  void* y;               // T or (out_f32) float [M][ldy]
  int ldy, out_f32;
  DenseOut out;          // STORE
  float limit;                        // GLU
  float* state;                       // MINGRU: [slots][N]
  const int32_t *pos, *seq;           // MINGRU: [M]
  unsigned long long* key;            // LOGITS: [M]
};
int jg_dense_call(jg_dev* dev, const DenseCall& c);
// bf16, any row count, tcgen05 (epilogues STORE and GLU)
int jg_dense_tc(jg_dev* dev, const DenseCall& c);
