// Linear recurrences with a matrix state per head, S <- a S + b k v^T and o = S^T q: a constant decay per head, or the
// exponential gates of mLSTM with its normaliser (jg_linear_desc).  What follows them — division, norm over groups of
// heads, output gate — is gated_row (stream.cuh), in the projection that comes next or in jg_gated_norm.
//
//   linear_step    one token per row: a CTA takes 32 columns of a head's state
//   linear_gates   gated portions: running maximum and the tokens' weights, one CTA per head of a sequence
//   linear_scan    portions token by token, 32 columns per CTA (fp32, short portions, odd sizes)
//   linear_chunk   bf16 portions, 64 tokens at a time on the tensor cores
//
// State, gates and weights are fp32.  On the tensor cores every fp32 operand (state, weights, weighted values) enters as two
// bf16 numbers, its rounding and what that left over, so that a product keeps 16 bits; q, k and v are bf16 to begin with.
// The normaliser is one more column of the state, with 1 in place of v.
#include <stddef.h>

#include "mma.cuh"

template <typename T>
struct LinArgs {
  const T *q, *k, *v;
  const float *gates, *decay;
  float *state, *m, *o, *den;
  float4* tok;  // gated portions, [R][H]: see linear_gates
  const int32_t *pos, *seq;
  int B, Sc, H, dim, vd, cols, ldp, lds;
  float q_scale, cap;
};

__device__ __forceinline__ float2 linear_gate(const float* z, int h, int H, float cap) {  // log input gate, log forget gate
  return make_float2(cap * tanhf(z[h] / cap), log_sigmoid_f32(cap * tanhf(z[H + h] / cap)));
}
__device__ __forceinline__ float linear_den(float x, float m) { return fmaxf(fabsf(x), expf(-m)) + 1e-6f; }

// One column of S, spread over 8 lanes, E elements each: lane l holds the float4s l, l + 8, l + 16, ...
constexpr int LI_LPC = 8, LI_THREADS = 256, LI_COLS = LI_THREADS / LI_LPC;
template <int E>
struct LinCol {
  float s[E];
  __device__ __forceinline__ void load(const float* p, int l, int lds, bool live) {
#pragma unroll
    for (int i = 0; i < E / 4; i++) {
      const int off = (l + LI_LPC * i) * 4;
      const float4 v = (live && off < lds) ? *reinterpret_cast<const float4*>(p + off) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[4 * i] = v.x; s[4 * i + 1] = v.y; s[4 * i + 2] = v.z; s[4 * i + 3] = v.w;
    }
  }
  __device__ __forceinline__ void store(float* p, int l, int lds) const {
#pragma unroll
    for (int i = 0; i < E / 4; i++) {
      const int off = (l + LI_LPC * i) * 4;
      if (off < lds) *reinterpret_cast<float4*>(p + off) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
    }
  }
  // one token; returns this lane's part of S^T q.  k and q: rows in shared memory, zeros past the head
  __device__ __forceinline__ float step(const float* k, const float* q, int l, float a, float bv) {
    float acc[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < E / 4; i++) {
      const float4 kv = *reinterpret_cast<const float4*>(k + (l + LI_LPC * i) * 4), qv = *reinterpret_cast<const float4*>(q + (l + LI_LPC * i) * 4);
      s[4 * i] = fmaf(kv.x, bv, a * s[4 * i]);
      s[4 * i + 1] = fmaf(kv.y, bv, a * s[4 * i + 1]);
      s[4 * i + 2] = fmaf(kv.z, bv, a * s[4 * i + 2]);
      s[4 * i + 3] = fmaf(kv.w, bv, a * s[4 * i + 3]);
      acc[0] = fmaf(s[4 * i], qv.x, acc[0]);
      acc[1] = fmaf(s[4 * i + 1], qv.y, acc[1]);
      acc[0] = fmaf(s[4 * i + 2], qv.z, acc[0]);
      acc[1] = fmaf(s[4 * i + 3], qv.w, acc[1]);
    }
    return acc[0] + acc[1];
  }
};
__device__ __forceinline__ float sum_lanes8(float v) {
#pragma unroll
  for (int o = LI_LPC / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

template <typename T, int E>
__global__ void __launch_bounds__(LI_THREADS) linear_step_kernel(const LinArgs<T> a) {
  constexpr int DP = E * LI_LPC;
  __shared__ __align__(16) float sk[DP], sq[DP];
  pdl_launch();
  const int tid = threadIdx.x, l = tid % LI_LPC, h = blockIdx.y, r = blockIdx.z, c = blockIdx.x * LI_COLS + tid / LI_LPC;
  pdl_wait();
  const int p0 = a.pos[r], slot = a.seq[r];
  const bool live = c < a.cols;
  float* st = a.state + (((size_t)slot * a.H + h) * a.cols + min(c, a.cols - 1)) * a.lds;
  LinCol<E> S;
  S.load(st, l, a.lds, p0 > 0);
  float ad, b = 1.f, m = 0.f;
  if (a.gates) {
    const float m0 = p0 > 0 ? a.m[((size_t)slot * 2 + (p0 & 1)) * a.H + h] : 0.f;
    const float2 g = linear_gate(a.gates + (size_t)r * 2 * a.H, h, a.H, a.cap);
    m = fmaxf(g.y + m0, g.x);
    ad = expf(g.y + m0 - m);
    b = expf(g.x - m);
  } else {
    ad = a.decay[h];
  }
  for (int i = tid; i < DP; i += LI_THREADS) {
    const size_t at = (size_t)r * a.ldp + h * a.dim + i;
    sk[i] = i < a.dim ? to_f32(a.k[at]) : 0.f;
    sq[i] = i < a.dim ? to_f32(a.q[at]) * a.q_scale : 0.f;
  }
  const float v = c < a.vd ? to_f32(a.v[(size_t)r * a.ldp + h * a.vd + c]) : 1.f;
  __syncthreads();
  const float x = sum_lanes8(S.step(sk, sq, l, ad, b * v));
  if (!live) return;
  S.store(st, l, a.lds);
  if (l != 0) return;
  if (c < a.vd) {
    a.o[((size_t)r * a.H + h) * a.vd + c] = x;
  } else {
    a.den[(size_t)r * a.H + h] = linear_den(x, m);
    a.m[((size_t)slot * 2 + ((p0 + 1) & 1)) * a.H + h] = m;  // the other entry: no CTA of this step reads it
  }
}

// Weights of a gated portion, per token and head: with b_t the sum of the log forget gates since the start of the token's
// block of `block` tokens, (b_t - m_t, i_t - b_t, m_t, m_{t-1}) with the first two in powers of two; with block = 0 (a_t, b_t, m_t, -) of the recurrence.
// m_t = max(f_t + m_{t-1}, i_t) is a map of m_{t-1}; maps compose, (F1, I1) then (F2, I2) = (F1 + F2, max(F2 + I1, I2)).
constexpr int LG_THREADS = 1024;
__device__ __forceinline__ void scan_max_plus(float& F, float& I, int lane) {  // inclusive, over the lanes of a warp
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float f1 = __shfl_up_sync(0xffffffffu, F, o), i1 = __shfl_up_sync(0xffffffffu, I, o);
    if (lane >= o) { I = fmaxf(F + i1, I); F += f1; }
  }
}
__global__ void __launch_bounds__(LG_THREADS) linear_gates_kernel(const float* __restrict__ gates, float* __restrict__ m_state, float4* __restrict__ tok, const int32_t* __restrict__ pos,
                                                                  const int32_t* __restrict__ seq, int B, int Sc, int H, float cap, int block) {
  __shared__ float2 s_warp[2][LG_THREADS / 32];  // the warps' maps, two blocks in turn
  pdl_launch();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, b = blockIdx.y, p0 = pos[b];
  float* ms = m_state + (size_t)seq[b] * 2 * H + h;
  float carry = p0 > 0 ? ms[(size_t)(p0 & 1) * H] : 0.f;
  auto gate = [&](int t) { return t < Sc ? linear_gate(gates + ((size_t)t * B + b) * 2 * H, h, H, cap) : make_float2(-INFINITY, 0.f); };  // past the end: the identity
  float2 g = gate(tid);
  for (int t0 = 0, buf = 0; t0 < Sc; t0 += LG_THREADS, buf ^= 1) {
    const int t = t0 + tid;
    float F = g.y, I = g.x;
    scan_max_plus(F, I, lane);
    if (lane == 31) s_warp[buf][warp] = make_float2(F, I);
    const float2 next = gate(t + LG_THREADS);
    __syncthreads();
    float2 w = s_warp[buf][lane];  // one map per warp: every warp runs through them itself
    const float before_me = block > 0 && (warp & 1) ? s_warp[buf][warp - 1].x : 0.f;
    scan_max_plus(w.x, w.y, lane);
    const float ends = fmaxf(w.x + carry, w.y);  // lane l: the maximum after warp l
    const float ahead = __shfl_sync(0xffffffffu, ends, max(warp - 1, 0)), start = warp > 0 ? ahead : carry;
    const float m = fmaxf(F + start, I), up = __shfl_up_sync(0xffffffffu, m, 1), before = lane > 0 ? up : start;
    const float bt = F + before_me;  // blocks of 64 tokens: two warps
    if (t < Sc)
      tok[((size_t)t * B + b) * H + h] = block > 0 ? make_float4((bt - m) * LOG2E, (g.x - bt) * LOG2E, m, before) : make_float4(expf(g.y + before - m), expf(g.x - m), m, 0.f);
    carry = __shfl_sync(0xffffffffu, ends, LG_THREADS / 32 - 1);
    g = next;
  }
  if (tid == 0) ms[(size_t)((p0 + Sc) & 1) * H] = carry;
}

constexpr int LN_TOK = 16;
template <typename T, int E>
__global__ void __launch_bounds__(LI_THREADS) linear_scan_kernel(const LinArgs<T> a) {
  constexpr int DP = E * LI_LPC;
  extern __shared__ __align__(16) float sm[];
  float *sk = sm, *sq = sk + LN_TOK * DP, *sv = sq + LN_TOK * DP, *sa = sv + LN_TOK * LI_COLS, *sb = sa + LN_TOK, *s_max = sb + LN_TOK;
  pdl_wait();
  const int tid = threadIdx.x, l = tid % LI_LPC, cl = tid / LI_LPC, h = blockIdx.y, b = blockIdx.z, c = blockIdx.x * LI_COLS + cl;
  const int slot = a.seq[b];
  const bool live = c < a.cols;
  float* st = a.state + (((size_t)slot * a.H + h) * a.cols + min(c, a.cols - 1)) * a.lds;
  LinCol<E> S;
  S.load(st, l, a.lds, a.pos[b] > 0);
  for (int t0 = 0; t0 < a.Sc; t0 += LN_TOK) {
    const int nt = min(LN_TOK, a.Sc - t0);
    __syncthreads();
    for (int i = tid; i < nt * DP; i += LI_THREADS) {
      const int t = i / DP, e = i % DP;
      const size_t at = ((size_t)(t0 + t) * a.B + b) * a.ldp + h * a.dim + e;
      sk[i] = e < a.dim ? to_f32(a.k[at]) : 0.f;
      sq[i] = e < a.dim ? to_f32(a.q[at]) * a.q_scale : 0.f;
    }
    for (int i = tid; i < nt * LI_COLS; i += LI_THREADS) {
      const int t = i / LI_COLS, cc = blockIdx.x * LI_COLS + i % LI_COLS;
      sv[i] = cc < a.vd ? to_f32(a.v[((size_t)(t0 + t) * a.B + b) * a.ldp + h * a.vd + cc]) : 1.f;
    }
    if (tid < nt) {
      const float4 g = a.gates ? a.tok[((size_t)(t0 + tid) * a.B + b) * a.H + h] : make_float4(a.decay[h], 1.f, 0.f, 0.f);
      sa[tid] = g.x; sb[tid] = g.y; s_max[tid] = g.z;
    }
    __syncthreads();
    for (int t = 0; t < nt; t++) {
      const float x = sum_lanes8(S.step(sk + t * DP, sq + t * DP, l, sa[t], sb[t] * sv[t * LI_COLS + cl]));
      if (l != 0 || !live) continue;
      const size_t r = (size_t)(t0 + t) * a.B + b;
      if (c < a.vd) a.o[(r * a.H + h) * a.vd + c] = x;
      else a.den[r * a.H + h] = linear_den(x, s_max[t]);
    }
  }
  pdl_launch();
  if (live) S.store(st, l, a.lds);
}

// ------------------------------------------------------------------------------------------------ tensor cores
// A CTA keeps 32 columns of a head's state, transposed, in the accumulators of its eight warps (16 columns x a quarter of the
// head each) and walks the sequence 64 tokens at a time.  With D the tokens' weights (jg_linear_desc, products of decays),
//   A[t][s]  = D[t][s] (k_s . q_t) for s <= t                    q, k in shared memory, two warps per 16 rows
//   O^T      = (S^T q_t) dec_t + V^T A^T                          S^T straight from the accumulators as A fragments
//   S^T      = g S^T + (w V)^T K
// The quarters of the head add up their O^T through shared memory.
constexpr int LK_TOK = 64, LK_COLS = 32, LK_WARPS = 8, LK_THREADS = 32 * LK_WARPS, LK_LDA = LK_TOK + 8, LK_LDV = LK_COLS + 8, LK_LDR = LK_COLS + 4;
template <int DP>
struct LinStage {
  bf16 q[LK_TOK][DP + 8], k[LK_TOK][DP + 8], v[LK_TOK][LK_LDV];
  float4 g[LK_TOK];
};
template <int DP>
struct LinShared {
  LinStage<DP> st[2];
  bf16 hi[LK_TOK][LK_LDA], lo[LK_TOK][LK_LDA];
  float red[4][LK_TOK][LK_LDR];
  float dec[LK_TOK], w[LK_TOK], pw[LK_TOK + 1];
};
// 16-byte pieces in the stages, pairs of 8 bytes among the factors
static_assert(offsetof(LinStage<64>, g) % 16 == 0 && sizeof(LinStage<64>) % 16 == 0 && sizeof(LinStage<128>) % 16 == 0 && sizeof(LinStage<256>) % 16 == 0, "stage layout");
static_assert(offsetof(LinShared<64>, hi) % 16 == 0 && offsetof(LinShared<64>, lo) % 16 == 0 , "weight layout");
static_assert(offsetof(LinShared<64>, dec) % 8 == 0 && offsetof(LinShared<64>, w) % 8 == 0, "factor layout");

template <int DP, bool GATED>
__global__ void __launch_bounds__(LK_THREADS) linear_chunk_kernel(const LinArgs<bf16> a) {
  constexpr int NT = DP / 32;  // 8-wide tiles of a warp's quarter of the head
  extern __shared__ __align__(16) unsigned char lk_smem[];
  LinShared<DP>& sh = *reinterpret_cast<LinShared<DP>*>(lk_smem);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3, cg = warp & 1, dq = warp >> 1;
  const int h = blockIdx.y, b = blockIdx.z, j0 = blockIdx.x * LK_COLS;
  const int dpc = a.dim / 8;
  {  // what no load fills: past the head, and past the values (the normaliser's column holds ones)
    if (a.dim < DP)
      for (int i = tid; i < (int)(sizeof(sh.st) / 16); i += LK_THREADS) reinterpret_cast<uint4*>(sh.st)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();
    for (int i = tid; i < 2 * LK_TOK * (LK_COLS / 8); i += LK_THREADS) {
      const int c = i % (LK_COLS / 8) * 8;
      if (j0 + c >= a.vd) *reinterpret_cast<uint4*>(&sh.st[i / (LK_TOK * LK_COLS / 8)].v[i / (LK_COLS / 8) % LK_TOK][c]) = make_uint4(GATED && j0 + c == a.vd ? 0x3F80u : 0u, 0, 0, 0);
    }
  }
  pdl_wait();
  if (!GATED && tid <= LK_TOK) sh.pw[tid] = tid == 0 ? 1.f : powf(a.decay[h], (float)tid);
  // a warp brings every eighth token; a lane the same 16-byte pieces of each: where they come from and where they go
  constexpr int NP = (DP / 4 + LK_COLS / 8 + 31) / 32;
  const bf16* src[NP];
  uint32_t dst[NP], step[NP];  // bytes from the start of a stage, and between its tokens
#pragma unroll
  for (int n = 0; n < NP; n++) {
    const int c = lane + 32 * n, kc = c - dpc, vc = c - 2 * dpc;
    const size_t row = ((size_t)warp * a.B + b) * a.ldp;
    src[n] = nullptr;
    dst[n] = step[n] = 0;
    if (c < dpc) { src[n] = a.q + row + h * a.dim + c * 8; dst[n] = offsetof(LinStage<DP>, q) + c * 16; step[n] = sizeof(sh.st[0].q[0]); }
    else if (kc < dpc) { src[n] = a.k + row + h * a.dim + kc * 8; dst[n] = offsetof(LinStage<DP>, k) + kc * 16; step[n] = sizeof(sh.st[0].k[0]); }
    else if (vc < LK_COLS / 8 && j0 + vc * 8 < a.vd) { src[n] = a.v + row + h * a.vd + j0 + vc * 8; dst[n] = offsetof(LinStage<DP>, v) + vc * 16; step[n] = sizeof(sh.st[0].v[0]); }
    dst[n] += warp * step[n];
  }
  const size_t token = (size_t)a.B * a.ldp;
  auto load = [&](int t0, int s) {
    unsigned char* st = reinterpret_cast<unsigned char*>(&sh.st[s]);
    const int nt = a.Sc - t0;
#pragma unroll
    for (int n = 0; n < NP; n++)
      if (src[n]) {
        const bf16* p = src[n] + (size_t)t0 * token;
#pragma unroll
        for (int i = 0; i < LK_TOK / LK_WARPS; i++) {
          unsigned char* d = st + dst[n] + i * LK_WARPS * step[n];
          if (warp + i * LK_WARPS < nt) cp16(d, p + (size_t)i * LK_WARPS * token);
          else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);  // past the end
        }
      }
    if (GATED && tid < min(LK_TOK, nt)) cp16(&sh.st[s].g[tid], a.tok + ((size_t)(t0 + tid) * a.B + b) * a.H + h);
    cp_commit();
  };
  load(0, 0);
  float S[NT][4];
  const bool cont = a.pos[b] > 0;
  const int d0 = dq * (DP / 4), c0 = j0 + cg * 16 + g;
  float* state = a.state + ((size_t)a.seq[b] * a.H + h) * a.cols * a.lds;
#pragma unroll
  for (int j = 0; j < NT; j++)
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int c = c0 + 8 * i, d = d0 + j * 8 + tq * 2;
      const float2 v = cont && c < a.cols && d < a.lds ? *reinterpret_cast<const float2*>(state + (size_t)c * a.lds + d) : make_float2(0.f, 0.f);
      S[j][2 * i] = v.x; S[j][2 * i + 1] = v.y;
    }
  int s = 0;
  for (int t0 = 0; t0 < a.Sc; t0 += LK_TOK, s ^= 1) {
    const int nt = min(LK_TOK, a.Sc - t0);
    cp_wait<0>();
    __syncthreads();
    if (t0 + LK_TOK < a.Sc) load(t0 + LK_TOK, s ^ 1);
    LinStage<DP>& st = sh.st[s];
    float decay;  // of the state over the whole block
    {
      const float4 last = GATED ? st.g[nt - 1] : make_float4(0.f, 0.f, 0.f, 0.f);
      const float mp = GATED ? st.g[0].w * LOG2E : 0.f;
      decay = GATED ? ex2(last.x + mp) : sh.pw[nt];
      if (tid < LK_TOK) {
        const bool in = tid < nt;
        sh.dec[tid] = !in ? 0.f : a.q_scale * (GATED ? ex2(st.g[tid].x + mp) : sh.pw[tid + 1]);
        sh.w[tid] = !in ? 0.f : GATED ? ex2(last.x + st.g[tid].y) : sh.pw[nt - 1 - tid];
      }
    }
    {  // A: 16 tokens against the tokens up to them, every other pair of tiles
      const int rg = warp & 3, half = warp >> 2;
      float sc[2][2][4];
#pragma unroll
      for (int j = 0; j < 2; j++)
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
          for (int i = 0; i < 4; i++) sc[j][n][i] = 0.f;
      if (half <= rg) {
#pragma unroll 4
        for (int k = 0; k < DP; k += 16) {
          uint32_t qf[4];
          ldsm4(qf, &st.q[rg * 16 + (lane & 15)][k + (lane >> 4) * 8]);
#pragma unroll
          for (int j = 0; j < 2; j++)
            if (2 * j + half <= rg) {
              uint32_t kf[4];
              ldsm4(kf, &st.k[(2 * j + half) * 16 + (lane >> 4) * 8 + (lane & 7)][k + ((lane >> 3) & 1) * 8]);
              mma_bf16(sc[j][0], qf, kf[0], kf[1]);
              mma_bf16(sc[j][1], qf, kf[2], kf[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 2; j++)
          if (2 * j + half <= rg)
#pragma unroll
            for (int n = 0; n < 2; n++)
#pragma unroll
              for (int i = 0; i < 2; i++) {
                const int t = rg * 16 + g + 8 * i, e = (2 * j + half) * 16 + n * 8 + tq * 2;
                float x[2];
#pragma unroll
                for (int k = 0; k < 2; k++) {  // a later token has no weight, however far its exponent goes
                  const float w = GATED ? ex2(st.g[t].x + st.g[e + k].y) : sh.pw[max(t - e - k, 0)];
                  x[k] = e + k <= t && t < nt ? sc[j][n][2 * i + k] * (w * a.q_scale) : 0.f;
                }
                uint32_t hi, lo;
                split_bf16(x[0], x[1], hi, lo);
                *reinterpret_cast<uint32_t*>(&sh.hi[t][e]) = hi;
                *reinterpret_cast<uint32_t*>(&sh.lo[t][e]) = lo;
              }
      }
    }
    float o[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) o[j][i] = 0.f;
    // S^T q over this warp's quarter of the head
#pragma unroll
    for (int k = 0; k < NT / 2; k++) {
      uint32_t hi[4], lo[4], qf[4][4];
#pragma unroll
      for (int j = 0; j < 4; j++) ldsm4(qf[j], &st.q[j * 16 + (lane >> 4) * 8 + (lane & 7)][d0 + k * 16 + ((lane >> 3) & 1) * 8]);
      split_bf16(S[2 * k][0], S[2 * k][1], hi[0], lo[0]);
      split_bf16(S[2 * k][2], S[2 * k][3], hi[1], lo[1]);
      split_bf16(S[2 * k + 1][0], S[2 * k + 1][1], hi[2], lo[2]);
      split_bf16(S[2 * k + 1][2], S[2 * k + 1][3], hi[3], lo[3]);
#pragma unroll
      for (int j = 0; j < 4; j++) { mma_bf16(o[2 * j], hi, qf[j][0], qf[j][1]); mma_bf16(o[2 * j + 1], hi, qf[j][2], qf[j][3]); }
#pragma unroll
      for (int j = 0; j < 4; j++) { mma_bf16(o[2 * j], lo, qf[j][0], qf[j][1]); mma_bf16(o[2 * j + 1], lo, qf[j][2], qf[j][3]); }
    }
    __syncthreads();  // A, the decays and the weights are there
#pragma unroll
    for (int j = 0; j < 8; j++) {
      const float2 d = *reinterpret_cast<const float2*>(&sh.dec[j * 8 + tq * 2]);
      o[j][0] *= d.x; o[j][1] *= d.y; o[j][2] *= d.x; o[j][3] *= d.y;
    }
    {  // V^T A^T over this warp's quarter of the block's tokens
      uint32_t vf[4];
      ldsm4t(vf, &st.v[dq * 16 + (lane >> 4) * 8 + (lane & 7)][cg * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
      for (int j = 0; j < 4; j++)
        if (dq <= j) {
          uint32_t hi[4], lo[4];
          ldsm4(hi, &sh.hi[j * 16 + (lane >> 4) * 8 + (lane & 7)][dq * 16 + ((lane >> 3) & 1) * 8]);
          ldsm4(lo, &sh.lo[j * 16 + (lane >> 4) * 8 + (lane & 7)][dq * 16 + ((lane >> 3) & 1) * 8]);
          mma_bf16(o[2 * j], vf, hi[0], hi[1]);
          mma_bf16(o[2 * j + 1], vf, hi[2], hi[3]);
          mma_bf16(o[2 * j], vf, lo[0], lo[1]);
          mma_bf16(o[2 * j + 1], vf, lo[2], lo[3]);
        }
    }
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) sh.red[dq][j * 8 + tq * 2 + (i & 1)][cg * 16 + g + 8 * (i >> 1)] = o[j][i];
    // the state moves on by the block
#pragma unroll
    for (int j = 0; j < NT; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) S[j][i] *= decay;
#pragma unroll
    for (int ks = 0; ks < LK_TOK / 16; ks++) {
      uint32_t vf[4], hi[4], lo[4], kf[NT / 2][4];
      ldsm4t(vf, &st.v[ks * 16 + (lane >> 4) * 8 + (lane & 7)][cg * 16 + ((lane >> 3) & 1) * 8]);
#pragma unroll
      for (int j = 0; j < NT / 2; j++) ldsm4t(kf[j], &st.k[ks * 16 + (lane & 15)][d0 + j * 16 + (lane >> 4) * 8]);
      const float2 w0 = *reinterpret_cast<const float2*>(&sh.w[ks * 16 + tq * 2]), w1 = *reinterpret_cast<const float2*>(&sh.w[ks * 16 + 8 + tq * 2]);
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const float2 w = i < 2 ? w0 : w1;
        split_bf16(__uint_as_float(vf[i] << 16) * w.x, __uint_as_float(vf[i] & 0xFFFF0000u) * w.y, hi[i], lo[i]);
      }
#pragma unroll
      for (int j = 0; j < NT / 2; j++) { mma_bf16(S[2 * j], hi, kf[j][0], kf[j][1]); mma_bf16(S[2 * j + 1], hi, kf[j][2], kf[j][3]); }
#pragma unroll
      for (int j = 0; j < NT / 2; j++) { mma_bf16(S[2 * j], lo, kf[j][0], kf[j][1]); mma_bf16(S[2 * j + 1], lo, kf[j][2], kf[j][3]); }
    }
    __syncthreads();
    const int c = j0 + lane;  // a warp writes 32 columns of a token
    if (c < a.cols)
#pragma unroll 2
      for (int t = warp; t < nt; t += LK_WARPS) {
        const float x = sh.red[0][t][lane] + sh.red[1][t][lane] + sh.red[2][t][lane] + sh.red[3][t][lane];
        const size_t r = (size_t)(t0 + t) * a.B + b;
        if (c < a.vd) a.o[(r * a.H + h) * a.vd + c] = x;
        else a.den[r * a.H + h] = linear_den(x, st.g[t].z);
      }
  }
  pdl_launch();
#pragma unroll
  for (int j = 0; j < NT; j++)
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int c = c0 + 8 * i, d = d0 + j * 8 + tq * 2;
      if (c < a.cols && d < a.lds) *reinterpret_cast<float2*>(state + (size_t)c * a.lds + d) = make_float2(S[j][2 * i], S[j][2 * i + 1]);
    }
}

// ------------------------------------------------------------------------------------------------ host side
constexpr int LINEAR_MIN_CHUNK = 16, LINEAR_MAX_DIM = 1024;

JG_API int jg_linear_scratch_bytes(const jg_linear_desc* d, int32_t rows, uint64_t* out) {
  JG_REQUIRE(d != nullptr && out != nullptr && rows > 0, "linear_scratch_bytes: bad arguments");
  *out = (uint64_t)rows * d->heads * sizeof(float4);
  return JG_OK;
}

template <typename T, int E>
static int linear_launch(jg_dev* dev, const LinArgs<T>& a) {
  const dim3 grid((unsigned)((a.cols + LI_COLS - 1) / LI_COLS), (unsigned)a.H, (unsigned)a.B);
  if (a.Sc == 1) return jg_launch(dev, "linear_step", linear_step_kernel<T, E>, grid, dim3(LI_THREADS), 0, a);
  constexpr size_t smem = (size_t)LN_TOK * (2 * E * LI_LPC + LI_COLS + 3) * sizeof(float);
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(linear_scan_kernel<T, E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    set[dev->ordinal & 7] = true;
  }
  return jg_launch(dev, "linear_scan", linear_scan_kernel<T, E>, grid, dim3(LI_THREADS), smem, a);
}
template <int DP, bool GATED>
static int launch_chunk(jg_dev* dev, const LinArgs<bf16>& a) {
  auto kern = linear_chunk_kernel<DP, GATED>;
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(LinShared<DP>)));
    set[dev->ordinal & 7] = true;
  }
  return jg_launch(dev, "linear_chunk", kern, dim3((unsigned)((a.cols + LK_COLS - 1) / LK_COLS), (unsigned)a.H, (unsigned)a.B), dim3(LK_THREADS), sizeof(LinShared<DP>), a);
}
// whether a portion runs on the tensor cores
static bool chunkable(const LinArgs<float>&) { return false; }
static bool chunkable(const LinArgs<bf16>& a) {
  return a.Sc >= LINEAR_MIN_CHUNK && a.dim % 8 == 0 && a.vd % 8 == 0 && a.dim <= 256 && a.ldp % 8 == 0 && (uintptr_t)a.q % 16 == 0 && (uintptr_t)a.k % 16 == 0 && (uintptr_t)a.v % 16 == 0;
}
static int run_chunk(jg_dev*, const LinArgs<float>&) { return JG_ENOTSUP; }
static int run_chunk(jg_dev* dev, const LinArgs<bf16>& a) {
  if (a.dim <= 64) return a.gates ? launch_chunk<64, true>(dev, a) : launch_chunk<64, false>(dev, a);
  if (a.dim <= 128) return a.gates ? launch_chunk<128, true>(dev, a) : launch_chunk<128, false>(dev, a);
  return a.gates ? launch_chunk<256, true>(dev, a) : launch_chunk<256, false>(dev, a);
}

template <typename T>
static int linear_run(jg_dev* dev, const jg_batch* b, const jg_linear_desc* d) {
  LinArgs<T> a = {};
  a.q = (const T*)d->q; a.k = (const T*)d->k; a.v = (const T*)d->v; a.gates = (const float*)d->gates; a.decay = (const float*)d->decay;
  a.state = (float*)d->state; a.m = (float*)d->m; a.o = (float*)d->o; a.den = (float*)d->den; a.tok = (float4*)d->scratch;
  a.pos = (const int32_t*)b->pos; a.seq = (const int32_t*)b->seq;
  a.B = b->B; a.Sc = b->Sc; a.H = d->heads; a.dim = d->dim; a.vd = d->vdim; a.cols = d->vdim + (d->gates ? 1 : 0); a.ldp = d->ldp;
  a.lds = (d->dim + 3) & ~3; a.q_scale = d->q_scale; a.cap = d->cap;
  const bool chunk = chunkable(a);
  if (a.gates && a.Sc > 1) {
    int rc = jg_launch(dev, "linear_gates", linear_gates_kernel, dim3((unsigned)a.H, (unsigned)a.B), dim3(LG_THREADS), 0, a.gates, a.m, a.tok, a.pos, a.seq, a.B, a.Sc, a.H, a.cap,
                       chunk ? LK_TOK : 0);
    if (rc) return rc;
  }
  if (chunk) return run_chunk(dev, a);
  if (d->dim <= 32) return linear_launch<T, 4>(dev, a);
  if (d->dim <= 64) return linear_launch<T, 8>(dev, a);
  if (d->dim <= 128) return linear_launch<T, 16>(dev, a);
  if (d->dim <= 256) return linear_launch<T, 32>(dev, a);
  if (d->dim <= 512) return linear_launch<T, 64>(dev, a);
  return linear_launch<T, 128>(dev, a);
}

JG_API int jg_linear_state(jg_dev* dev, const jg_batch* b, const jg_linear_desc* d) {
  JG_ENTER(dev);
  JG_REQUIRE(d != nullptr && b != nullptr && b->B > 0 && b->Sc > 0 && jg_aligned(b->pos, 4) && jg_aligned(b->seq, 4), "linear_state: bad batch");
  JG_REQUIRE(d->dtype == JG_F32 || d->dtype == JG_BF16, "linear_state: unknown element type %d", d->dtype);
  JG_REQUIRE(d->heads > 0 && d->heads <= 65535 && b->B <= 65535 && d->dim > 0 && d->vdim > 0 && d->ldp >= d->heads * (d->dim > d->vdim ? d->dim : d->vdim), "linear_state: bad shape");
  if (d->dim > LINEAR_MAX_DIM) { jg_set_error("linear_state: query / key heads of %d values (largest supported: %d)", d->dim, LINEAR_MAX_DIM); return JG_ENOTSUP; }
  JG_REQUIRE(d->q && d->k && d->v && jg_aligned(d->state, 16) && jg_aligned(d->o, 4), "linear_state: null or misaligned pointer");
  if (d->gates) JG_REQUIRE(jg_aligned(d->gates, 4) && jg_aligned(d->m, 4) && jg_aligned(d->den, 4) && jg_aligned(d->scratch, 16) && d->cap > 0.f, "linear_state: null or misaligned gate pointer");
  else JG_REQUIRE(jg_aligned(d->decay, 4), "linear_state: null or misaligned decay");
  return d->dtype == JG_F32 ? linear_run<float>(dev, b, d) : linear_run<bf16>(dev, b, d);
}
