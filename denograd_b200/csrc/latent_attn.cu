// Latent attention over a paged ring of (normed latent | rotated key part) rows: a sliding window, a learned sink in the
// softmax's denominator, YaRN-scaled half-split rotary on the shared key part.
//
//   absorbed (decoding, short portions, fp32): the per-head key and value projections are applied to the query and to the
//   attended latent instead of to every cached position
//       latent_pre      qt = [W_uk^T q_unrotated | rotated q] per head; norm, rotation and cache row of the new tokens
//       latent_mma      bf16: scores qt . cache row, softmax statistics and the weighted latent of a context slice, for 16
//                       or 32 heads at once on the tensor cores (all heads share the cached rows)
//       latent_split    the same for one head on the CUDA cores (fp32, and shapes the other does not take)
//       latent_combine  slices + sink -> latent, then W_uv
//   expanded (bf16 prompt portions): keys and values of the window and the new tokens are projected once
//       latent_write    cache rows of the new tokens, and the attended rows side by side in scratch
//       dense           [W_uk | W_uv] on those rows
//       latent_chunk    causal windowed attention, 64 queries of a head per CTA, one pass with running statistics
//
// Scores, softmax statistics and weights are fp32; on the tensor cores the weights meet the values in bf16.
#include <math.h>
#include <stdlib.h>

#include "dense.cuh"
#include "mma.cuh"

template <typename T>
struct LatentArgs {
  const T* proj;
  T* pool;
  const int32_t* bt;
  const float *rot, *norm_w, *sink;
  const T *uk, *uv;
  T* qt;        // [R][H][lq]
  float* part;  // [R][H][ns][lat4] weighted latents of the slices (lat4: the latent rounded up to 4)
  float2* stat;  // [R][H][ns] their maxima and sums
  T* ctx;       // expanded form: [B][T][ldc]
  const T* kv;  // [B][T][ldkv]: keys of all heads, then values
  T* out;
  const int32_t *pos, *seq;
  int B, Sc, H, dim, rd, vd, rank, window, ldp, ldo, ldc, ldu, page, page_shift, pps, rot_pairs, rot_rows, ns, lq, lat4;
  int slice_round;  // slices are multiples of this many positions
  int T_ctx, T_prev, start, ldkv;
  int shift;  // tokens of this call ahead of its first row (a portion worked off in several passes)
  float eps, scale;
  __device__ __forceinline__ int qk() const { return dim + rd; }
  __host__ __device__ __forceinline__ int lat() const { return rank + rd; }
  // cache row of position p of the slot whose block-table row is `t`
  __device__ __forceinline__ T* row(const int32_t* t, int p) const {
    return pool + ((size_t)t[(p >> page_shift) % pps] * page + (p & (page - 1))) * ldc;
  }
  // positions per slice when a row sees n of them
  __device__ __forceinline__ int slice(int n) const { return ((n + ns - 1) / ns + slice_round - 1) / slice_round * slice_round; }
  __device__ __forceinline__ int position(int r) const { return min(max(pos[r % B] + shift + r / B, 0), rot_rows - 1); }
};

// Entry i of a rotated vector: pairs (i, i + rot_pairs) turn, the rest passes.
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int i, const float* cs, int pairs) {
  if (i >= 2 * pairs) return to_f32(x[i]);
  const int j = i < pairs ? i : i - pairs;
  const float u = to_f32(x[j]), v = to_f32(x[j + pairs]), c = cs[2 * j], s = cs[2 * j + 1];
  return i < pairs ? fmaf(u, c, -v * s) : fmaf(v, c, u * s);
}

// Cache row of the new token in row r, by one warp; `copy` (or null) receives it too.  Up to 512 latent values stay in
// registers between the norm and the store, their loads all in flight at once.
template <typename T>
__device__ __forceinline__ void write_row(const LatentArgs<T>& a, int r, int lane, T* copy) {
  constexpr int KEEP = 16;
  const int b = r % a.B, p = a.pos[b] + a.shift + r / a.B;
  const T* c = a.proj + (size_t)r * a.ldp + a.H * a.qk();
  float v[KEEP], w[KEEP], ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; k++) {
    const int i = lane + 32 * k;
    v[k] = i < a.rank ? to_f32(c[i]) : 0.f;
    w[k] = i < a.rank ? a.norm_w[i] : 0.f;
  }
#pragma unroll
  for (int k = 0; k < KEEP; k++) ss = fmaf(v[k], v[k], ss);
  for (int i = lane + 32 * KEEP; i < a.rank; i += 32) { const float x = to_f32(c[i]); ss = fmaf(x, x, ss); }
  const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)a.rank + a.eps);
  if (p < 0 || p >= a.rot_rows) return;  // outside the tables: left alone
  T* dst = a.row(a.bt + (size_t)a.seq[b] * a.pps, p);
  auto put = [&](int i, float x) {
    const T t = from_f32<T>(x);
    dst[i] = t;
    if (copy) copy[i] = t;
  };
#pragma unroll
  for (int k = 0; k < KEEP; k++)
    if (lane + 32 * k < a.rank) put(lane + 32 * k, v[k] * rs * w[k]);
  for (int i = lane + 32 * KEEP; i < a.rank; i += 32) put(i, to_f32(c[i]) * rs * a.norm_w[i]);
  const float* cs = a.rot + (size_t)p * a.rot_pairs * 2;
  for (int i = lane; i < a.ldc - a.rank; i += 32) put(a.rank + i, i < a.rd ? rotated(c + a.rank, i, cs, a.rot_pairs) : 0.f);
}

template <typename T>
__global__ void __launch_bounds__(256) latent_write_kernel(const LatentArgs<T> a, int R) {
  pdl_wait();
  const int w = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (w < R) {
    write_row(a, w, lane, a.ctx + ((size_t)(w % a.B) * a.T_ctx + a.T_prev + w / a.B) * a.ldc);
  } else if (w < R + a.B * a.T_prev) {  // an earlier position that the window still reaches
    const int b = (w - R) / a.T_prev, j = (w - R) % a.T_prev;
    const uint4* src = reinterpret_cast<const uint4*>(a.row(a.bt + (size_t)a.seq[b] * a.pps, a.start - a.T_prev + j));
    uint4* dst = reinterpret_cast<uint4*>(a.ctx + ((size_t)b * a.T_ctx + j) * a.ldc);
    for (int i = lane; i < a.ldc / Elem<T>::VEC; i += 32) dst[i] = src[i];
  }
}

// ------------------------------------------------------------------------------------------------ absorbed form
constexpr int LP_COLS = 64;  // latent columns of a CTA; it serves LP_ROWS activation rows with one read of the weights

// Blocks 0 .. H * slices - 1: head and 64 latent columns of LP_ROWS rows; the last block along x writes those rows' cache
// rows.  All warps run down W_uk together, each thread a 16-byte piece of a row.
template <typename T, int LP_ROWS>
__global__ void __launch_bounds__(256) latent_pre_kernel(const LatentArgs<T> a, int R) {
  constexpr int VEC = Elem<T>::VEC, TPR = LP_COLS / VEC, DR = 256 / TPR, AHEAD = 4;
  extern __shared__ float sq[];  // [LP_ROWS][dim]
  __shared__ float red[8][LP_ROWS][LP_COLS];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r0 = blockIdx.y * LP_ROWS, nr = min(LP_ROWS, R - r0);
  pdl_launch();
  if (blockIdx.x == gridDim.x - 1) {
    pdl_wait();
    if (warp < nr) write_row(a, r0 + warp, lane, (T*)nullptr);
    return;
  }
  const int slices = (a.rank + LP_COLS - 1) / LP_COLS, h = blockIdx.x / slices, c0 = (blockIdx.x % slices) * LP_COLS;
  const int dr = tid / TPR, cc = c0 + (tid % TPR) * VEC;
  const T* uk = a.uk + (size_t)h * a.dim * a.ldu + cc;
  const bool in = cc < a.ldu;
  uint4 ahead[AHEAD];  // parameters: requested before the dependency wait
#pragma unroll
  for (int i = 0; i < AHEAD; i++) ahead[i] = (in && dr + i * DR < a.dim) ? ld_128(uk + (size_t)(dr + i * DR) * a.ldu) : make_uint4(0, 0, 0, 0);
  pdl_wait();
  for (int i = tid; i < LP_ROWS * a.dim; i += 256) {
    const int r = i / a.dim;
    sq[i] = r < nr ? to_f32(a.proj[(size_t)(r0 + r) * a.ldp + (size_t)h * a.qk() + i % a.dim]) : 0.f;
  }
  __syncthreads();
  float acc[LP_ROWS][VEC];
#pragma unroll
  for (int r = 0; r < LP_ROWS; r++)
#pragma unroll
    for (int k = 0; k < VEC; k++) acc[r][k] = 0.f;
  auto use = [&](const uint4& raw, int d) {
    float w[VEC];
    unpack_chunk(raw, w);
#pragma unroll
    for (int r = 0; r < LP_ROWS; r++) {
      const float q = sq[r * a.dim + d];
#pragma unroll
      for (int k = 0; k < VEC; k++) acc[r][k] = fmaf(q, w[k], acc[r][k]);
    }
  };
#pragma unroll
  for (int i = 0; i < AHEAD; i++)
    if (dr + i * DR < a.dim) use(ahead[i], dr + i * DR);
  for (int d = dr + AHEAD * DR; d < a.dim; d += DR)
    if (in) use(ld_128(uk + (size_t)d * a.ldu), d);
#pragma unroll
  for (int r = 0; r < LP_ROWS; r++)
#pragma unroll
    for (int k = 0; k < VEC; k++) {
      float v = acc[r][k];
#pragma unroll
      for (int o = TPR; o < 32; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if (lane < TPR) red[warp][r][lane * VEC + k] = v;
    }
  __syncthreads();
  for (int i = tid; i < nr * LP_COLS; i += 256) {
    const int r = i / LP_COLS, c = i % LP_COLS;
    if (c0 + c >= a.rank) continue;
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) v += red[w][r][c];
    a.qt[((size_t)(r0 + r) * a.H + h) * a.lq + c0 + c] = from_f32<T>(v);
  }
  if (c0 == 0) {  // the rotated part and the padding
    const int n = a.lq - a.rank;
    for (int i = tid; i < nr * n; i += 256) {
      const int r = i / n, e = i % n;
      const float* cs = a.rot + (size_t)a.position(r0 + r) * a.rot_pairs * 2;
      const T* q = a.proj + (size_t)(r0 + r) * a.ldp + (size_t)h * a.qk() + a.dim;
      a.qt[((size_t)(r0 + r) * a.H + h) * a.lq + a.rank + e] = from_f32<T>(e < a.rd ? rotated(q, e, cs, a.rot_pairs) : 0.f);
    }
  }
}

// The same for up to 16 rows on the tensor cores (bf16, three rows and more): [16 rows][dim] x [dim][64 latent columns].
constexpr int LPM_ROWS = 16, LPM_THREADS = 128;
static constexpr size_t lpm_smem(int dp) { return (size_t)2 * (dp * (LP_COLS + 8) + LPM_ROWS * (dp + 8)); }

__global__ void __launch_bounds__(LPM_THREADS) latent_pre_mma_kernel(const LatentArgs<bf16> a, int R, int dp) {
  extern __shared__ __align__(16) unsigned char smem[];
  bf16 *sW = reinterpret_cast<bf16*>(smem), *sQ = sW + (size_t)dp * (LP_COLS + 8);  // dp: dim rounded up to 16
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, r0 = blockIdx.y * LPM_ROWS, nr = min(LPM_ROWS, R - r0);
  pdl_launch();
  if (blockIdx.x >= gridDim.x - LPM_ROWS / 4) {  // the last blocks write the cache rows, one per warp
    const int r = (int)(blockIdx.x - (gridDim.x - LPM_ROWS / 4)) * 4 + warp;
    pdl_wait();
    if (r < nr) write_row(a, r0 + r, lane, (bf16*)nullptr);
    return;
  }
  const int slices = (a.rank + LP_COLS - 1) / LP_COLS, h = blockIdx.x / slices, c0 = (blockIdx.x % slices) * LP_COLS;
  for (int i = tid; i < dp * (LP_COLS / 8); i += LPM_THREADS) {  // parameters: ahead of the dependency wait
    const int d = i / (LP_COLS / 8), c = i % (LP_COLS / 8) * 8;
    bf16* dst = sW + (size_t)d * (LP_COLS + 8) + c;
    if (d < a.dim && c0 + c < a.ldu) cp16(dst, a.uk + ((size_t)h * a.dim + d) * a.ldu + c0 + c);
    else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
  }
  cp_commit();
  pdl_wait();
#pragma unroll
  for (int k = 0; k < LPM_ROWS / 4; k++) {
    const int r = k * 4 + warp;
    const bf16* src = a.proj + (size_t)(r0 + min(r, nr - 1)) * a.ldp + (size_t)h * a.qk();
#pragma unroll 4
    for (int d = lane; d < dp; d += 32) sQ[(size_t)r * (dp + 8) + d] = (r < nr && d < a.dim) ? src[d] : __float2bfloat16_rn(0.f);
  }
  cp_wait<0>();
  __syncthreads();
  float acc[2][4] = {};
  for (int k = 0; k < dp; k += 16) {
    uint32_t q[4], w[4];
    ldsm4(q, sQ + (size_t)(lane & 15) * (dp + 8) + k + (lane >> 4) * 8);
    ldsm4t(w, sW + (size_t)(k + (lane & 15)) * (LP_COLS + 8) + warp * 16 + (lane >> 4) * 8);
    mma_bf16(acc[0], q, w[0], w[1]);
    mma_bf16(acc[1], q, w[2], w[3]);
  }
  const int g = lane >> 2, tq = lane & 3;
#pragma unroll
  for (int j = 0; j < 2; j++)
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int r = g + 8 * (i >> 1), c = c0 + warp * 16 + j * 8 + tq * 2 + (i & 1);
      if (r < nr && c < a.rank) a.qt[((size_t)(r0 + r) * a.H + h) * a.lq + c] = __float2bfloat16_rn(acc[j][i]);
    }
  if (c0 == 0) {
    const int n = a.lq - a.rank;
    for (int i = tid; i < nr * n; i += LPM_THREADS) {
      const int r = i / n, e = i % n;
      const float* cs = a.rot + (size_t)a.position(r0 + r) * a.rot_pairs * 2;
      const bf16* q = a.proj + (size_t)(r0 + r) * a.ldp + (size_t)h * a.qk() + a.dim;
      a.qt[((size_t)(r0 + r) * a.H + h) * a.lq + a.rank + e] = from_f32<bf16>(e < a.rd ? rotated(q, e, cs, a.rot_pairs) : 0.f);
    }
  }
}

constexpr int LS_THREADS = 128, LS_TILE = 64, LS_MAX_RANK = 1024, LS_MAX_NS = 32;

template <typename T>
__global__ void __launch_bounds__(LS_THREADS) latent_split_kernel(const LatentArgs<T> a) {
  constexpr int NR = LS_MAX_RANK / LS_THREADS;
  extern __shared__ float sq[];  // qt of this (row, head)
  __shared__ float sc[LS_TILE];
  __shared__ const T* rows[LS_TILE];
  pdl_launch();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int r = blockIdx.x, h = blockIdx.y, p = a.position(r), L = a.lat();
  const int32_t* bt = a.bt + (size_t)a.seq[r % a.B] * a.pps;
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0, n = p + 1 - lo;
  const int chunk = a.slice(n), t0 = lo + blockIdx.z * chunk, t1 = min(p + 1, t0 + chunk);
  if (t0 >= t1) return;  // nobody reads an empty slice
  const size_t id = ((size_t)r * a.H + h) * a.ns + blockIdx.z;
  float* part = a.part + id * a.lat4;
  for (int i = tid; i < L; i += LS_THREADS) sq[i] = to_f32(a.qt[((size_t)r * a.H + h) * a.lq + i]);
  float acc[NR], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int k = 0; k < NR; k++) acc[k] = 0.f;
  for (int base = t0; base < t1; base += LS_TILE) {
    const int nt = min(LS_TILE, t1 - base);
    __syncthreads();
    if (tid < nt) rows[tid] = a.row(bt, base + tid);
    __syncthreads();
    for (int t = warp; t < nt; t += LS_THREADS / 32) {
      const T* c = rows[t];
      float d = 0.f;
      for (int i = lane; i < L; i += 32) d = fmaf(sq[i], to_f32(c[i]), d);
      d = warp_sum(d);
      if (lane == 0) sc[t] = d * a.scale;
    }
    __syncthreads();
    float mt = m;
    for (int t = 0; t < nt; t++) mt = fmaxf(mt, sc[t]);
    const float alpha = expf(m - mt);  // m = -inf on the first tile: 0
    m = mt;
    l *= alpha;
#pragma unroll
    for (int k = 0; k < NR; k++) acc[k] *= alpha;
    for (int t = 0; t < nt; t++) {
      const float e = expf(sc[t] - m);
      l += e;
      const T* c = rows[t];
#pragma unroll
      for (int k = 0; k < NR; k++)
        if (tid + k * LS_THREADS < a.rank) acc[k] = fmaf(e, to_f32(c[tid + k * LS_THREADS]), acc[k]);
    }
  }
  if (tid == 0) a.stat[id] = make_float2(m, l);
#pragma unroll
  for (int k = 0; k < NR; k++)
    if (tid + k * LS_THREADS < a.lat4) part[tid + k * LS_THREADS] = acc[k];  // zeros past the latent
}

// One row, 16 * MT heads, one context slice: tiles of 64 cached rows; a warp scores 16 of them for all heads over one part
// of the latent (NW / 4 partial score tiles), the heads' softmax statistics are dealt over the NW warps, and each warp owns
// NTW * 8 columns of the weighted latent.  A CTA fills an SM's shared memory: with 16 warps instead of 8 more of a tile's
// latencies overlap.
constexpr int LM_TILE = 64;
template <int MT, int NW>
static constexpr size_t lm_smem(int lq, int stages) {
  return (size_t)(stages * LM_TILE + 16 * MT) * (lq + 8) * 2 + (size_t)16 * MT * ((NW / 4) * LM_TILE * 4 + (LM_TILE + 8) * 2 + 12);
}

template <int MT, int NTW, int NW>
__global__ void __launch_bounds__(32 * NW) latent_mma_kernel(const LatentArgs<bf16> a, int stages) {
  extern __shared__ __align__(16) unsigned char smem[];
  constexpr int HR = 16 * MT, KS = NW / 4;
  const int ld = a.lq + 8;  // row stride: an odd number of 16-byte pieces
  bf16* tiles = reinterpret_cast<bf16*>(smem);
  bf16* sQ = tiles + (size_t)stages * LM_TILE * ld;
  float* sS = reinterpret_cast<float*>(sQ + (size_t)HR * ld);  // [KS][HR][64]
  bf16* sP = reinterpret_cast<bf16*>(sS + KS * HR * LM_TILE);  // [HR][72]
  float *sM = reinterpret_cast<float*>(sP + HR * (LM_TILE + 8)), *sL = sM + HR, *sA = sL + HR;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, z = blockIdx.x, h0 = blockIdx.y * HR, r = blockIdx.z;
  pdl_launch();
  pdl_wait();
  const int p = a.position(r);
  const int32_t* bt = a.bt + (size_t)a.seq[r % a.B] * a.pps;
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0, n = p + 1 - lo;
  const int chunk = a.slice(n), t0 = lo + z * chunk, t1 = min(p + 1, t0 + chunk);
  if (t0 >= t1) return;  // nobody reads an empty slice
  const int pieces = a.lq / 8, row_pieces = a.ldc / 8;
#pragma unroll
  for (int k = 0; k < HR / NW; k++) {  // a warp takes whole rows: one address calculation each
    const int h = k * NW + warp;
    const bf16* src = a.qt + ((size_t)r * a.H + min(h0 + h, a.H - 1)) * a.lq;
    for (int c = lane; c < pieces; c += 32) {
      bf16* d = sQ + (size_t)h * ld + c * 8;
      if (h0 + h < a.H) cp16(d, src + c * 8);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
    }
  }
  auto load_tile = [&](int base, int s) {
    bf16* t = tiles + (size_t)s * LM_TILE * ld;
    const bf16* src[LM_TILE / NW];
#pragma unroll
    for (int k = 0; k < LM_TILE / NW; k++) src[k] = a.row(bt, min(base + k * NW + warp, t1 - 1));
#pragma unroll
    for (int k = 0; k < LM_TILE / NW; k++) {
      const bool in = base + k * NW + warp < t1;
      bf16* d = t + (size_t)(k * NW + warp) * ld;
      for (int c = lane; c < pieces; c += 32) {
        if (in && c < row_pieces) cp16(d + c * 8, src[k] + c * 8);
        else *reinterpret_cast<uint4*>(d + c * 8) = make_uint4(0, 0, 0, 0);
      }
    }
    cp_commit();
  };
  load_tile(t0, 0);
  if (tid < HR) { sM[tid] = -INFINITY; sL[tid] = 0.f; }
  float o[MT][NTW][4];
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int j = 0; j < NTW; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) o[m][j][i] = 0.f;
  const int g = lane >> 2, tq = lane & 3;
  int s = 0;
  for (int base = t0; base < t1; base += LM_TILE) {
    const bool more = base + LM_TILE < t1;
    if (stages > 1 && more) { load_tile(base + LM_TILE, s ^ 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    const bf16* t = tiles + (size_t)s * LM_TILE * ld;
    float sc[MT][2][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int j = 0; j < 2; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) sc[m][j][i] = 0.f;
    const int pg = warp & 3, kh = warp >> 2;
    const bf16* kb = t + (size_t)(pg * 16 + (lane >> 4) * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8;
    const bf16* qb = sQ + (size_t)(lane & 15) * ld + (lane >> 4) * 8;
    const int k0 = a.lq / 16 * kh / KS * 16, k1 = a.lq / 16 * (kh + 1) / KS * 16;
#pragma unroll 2
    for (int k = k0; k < k1; k += 16) {
      uint32_t bk[4];
      ldsm4(bk, kb + k);
#pragma unroll
      for (int m = 0; m < MT; m++) {
        uint32_t q[4];
        ldsm4(q, qb + (size_t)m * 16 * ld + k);
        mma_bf16(sc[m][0], q, bk[0], bk[1]);
        mma_bf16(sc[m][1], q, bk[2], bk[3]);
      }
    }
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
      for (int j = 0; j < 2; j++)
#pragma unroll
        for (int i = 0; i < 2; i++) {
          const int c = pg * 16 + j * 8 + tq * 2;
          *reinterpret_cast<float2*>(sS + (size_t)kh * HR * LM_TILE + (m * 16 + g + 8 * i) * LM_TILE + c) =
              make_float2(base + c < t1 ? sc[m][j][2 * i] * a.scale : -INFINITY, base + c + 1 < t1 ? sc[m][j][2 * i + 1] * a.scale : -INFINITY);
        }
    __syncthreads();
    {  // the warp's heads side by side: their reductions overlap
      constexpr int NH = HR / NW;
      float x0[NH], x1[NH], old[NH], mx[NH], sum[NH];
#pragma unroll
      for (int k = 0; k < NH; k++) {
        const int row = k * NW + warp;
        x0[k] = x1[k] = 0.f;
#pragma unroll
        for (int q = 0; q < KS; q++) {
          x0[k] += sS[(q * HR + row) * LM_TILE + lane];
          x1[k] += sS[(q * HR + row) * LM_TILE + lane + 32];
        }
        old[k] = sM[row];
        mx[k] = fmaxf(x0[k], x1[k]);
      }
#pragma unroll
      for (int w = 16; w > 0; w >>= 1)
#pragma unroll
        for (int k = 0; k < NH; k++) mx[k] = fmaxf(mx[k], __shfl_xor_sync(0xffffffffu, mx[k], w));
#pragma unroll
      for (int k = 0; k < NH; k++) {
        mx[k] = fmaxf(mx[k], old[k]);
        x0[k] = expf(x0[k] - mx[k]);
        x1[k] = expf(x1[k] - mx[k]);
        sum[k] = x0[k] + x1[k];
      }
#pragma unroll
      for (int w = 16; w > 0; w >>= 1)
#pragma unroll
        for (int k = 0; k < NH; k++) sum[k] += __shfl_xor_sync(0xffffffffu, sum[k], w);
#pragma unroll
      for (int k = 0; k < NH; k++) {
        const int row = k * NW + warp;
        sP[row * (LM_TILE + 8) + lane] = __float2bfloat16_rn(x0[k]);
        sP[row * (LM_TILE + 8) + lane + 32] = __float2bfloat16_rn(x1[k]);
        if (lane == 0) {
          const float al = expf(old[k] - mx[k]);
          sA[row] = al;
          sL[row] = fmaf(sL[row], al, sum[k]);
          sM[row] = mx[k];
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; m++) {
      const float a0 = sA[m * 16 + g], a1 = sA[m * 16 + g + 8];
#pragma unroll
      for (int j = 0; j < NTW; j++) { o[m][j][0] *= a0; o[m][j][1] *= a0; o[m][j][2] *= a1; o[m][j][3] *= a1; }
    }
#pragma unroll
    for (int k = 0; k < LM_TILE; k += 16) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int m = 0; m < MT; m++) ldsm4(pf[m], sP + (size_t)(m * 16 + (lane & 15)) * (LM_TILE + 8) + k + (lane >> 4) * 8);
#pragma unroll
      for (int j = 0; j < NTW; j += 2) {
        const int c = (warp * NTW + j) * 8;
        if (c < a.rank) {  // a pair of column tiles may reach past the latent into the padding of the row, never past it
          uint32_t v[4];
          ldsm4t(v, t + (size_t)(k + (lane & 15)) * ld + c + (lane >> 4) * 8);
#pragma unroll
          for (int m = 0; m < MT; m++) {
            mma_bf16(o[m][j], pf[m], v[0], v[1]);
            mma_bf16(o[m][j + 1], pf[m], v[2], v[3]);
          }
        }
      }
    }
    __syncthreads();
    if (stages > 1) s ^= 1;
    else if (more) load_tile(base + LM_TILE, 0);
  }
  if (tid < HR && h0 + tid < a.H) a.stat[((size_t)r * a.H + h0 + tid) * a.ns + z] = make_float2(sM[tid], sL[tid]);
#pragma unroll
  for (int m = 0; m < MT; m++)
#pragma unroll
    for (int j = 0; j < NTW; j++)
#pragma unroll
      for (int i = 0; i < 2; i++) {
        const int h = h0 + m * 16 + g + 8 * i, c = (warp * NTW + j) * 8 + tq * 2;
        if (h < a.H && c < a.lat4) *reinterpret_cast<float2*>(a.part + (((size_t)r * a.H + h) * a.ns + z) * a.lat4 + c) = make_float2(o[m][j][2 * i], o[m][j][2 * i + 1]);
      }
}

// Slices and the sink -> the attended latent; then `outs` values of the head per CTA, for LC_ROWS rows.
constexpr int LC_ROWS = 4;
template <typename T>
__global__ void __launch_bounds__(256) latent_combine_kernel(const LatentArgs<T> a, int R, int outs) {
  constexpr int VEC = Elem<T>::VEC;
  extern __shared__ __align__(16) float so[];  // [LC_ROWS][lds] attended latents
  __shared__ float wgt[LC_ROWS][LS_MAX_NS];
  __shared__ int active[LC_ROWS];
  const int h = blockIdx.x, j0 = blockIdx.y * outs, j1 = min(a.vd, j0 + outs), r0 = blockIdx.z * LC_ROWS, nr = min(LC_ROWS, R - r0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, lds = (a.ldu + 3) & ~3;
  pdl_launch();
  // parameters: this warp's rows of W_uv travel to L2 while the predecessor drains
  for (int j = j0 + warp; j < j1; j += 8)
    for (size_t off = (size_t)lane * 128; off < (size_t)a.ldu * sizeof(T); off += 32 * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(a.uv + ((size_t)h * a.vd + j) * a.ldu) + off));
  pdl_wait();
  if (warp < nr) {
    const int p = a.position(r0 + warp), n = a.window > 0 ? min(p + 1, a.window) : p + 1, chunk = a.slice(n), na = (n + chunk - 1) / chunk;
    const float2 st = lane < na ? a.stat[((size_t)(r0 + warp) * a.H + h) * a.ns + lane] : make_float2(-INFINITY, 0.f);
    const float sink = a.sink[h], M = fmaxf(warp_max(st.x), sink), e = expf(st.x - M);
    const float L = warp_sum(st.y * e) + expf(sink - M);
    wgt[warp][lane] = e / L;
    if (lane == 0) active[warp] = na;
  }
  __syncthreads();
  for (int i = tid; i < nr * (lds / 4); i += 256) {
    const int r = i / (lds / 4), c = i % (lds / 4) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < a.lat4) {
      const float* part = a.part + ((size_t)(r0 + r) * a.H + h) * a.ns * a.lat4 + c;
      const int na = active[r];
#pragma unroll 8
      for (int s = 0; s < na; s++) {
        const float4 x = *reinterpret_cast<const float4*>(part + (size_t)s * a.lat4);
        const float w = wgt[r][s];
        v.x = fmaf(x.x, w, v.x); v.y = fmaf(x.y, w, v.y); v.z = fmaf(x.z, w, v.z); v.w = fmaf(x.w, w, v.w);
      }
    }
    *reinterpret_cast<float4*>(so + (size_t)r * lds + c) = v;  // what lies past the latent meets zeros of W_uv
  }
  __syncthreads();
  for (int j = j0 + warp; j < j1; j += 8) {
    const T* w = a.uv + ((size_t)h * a.vd + j) * a.ldu;
    float acc[LC_ROWS];
#pragma unroll
    for (int r = 0; r < LC_ROWS; r++) acc[r] = 0.f;
#pragma unroll 2
    for (int c = lane; c < a.ldu / VEC; c += 32) {
      float f[VEC];
      unpack_chunk(ld_128(w + (size_t)c * VEC), f);
#pragma unroll
      for (int r = 0; r < LC_ROWS; r++)
        if (r < nr) {
#pragma unroll
          for (int k = 0; k < VEC; k += 4) {
            const float4 x = *reinterpret_cast<const float4*>(so + (size_t)r * lds + c * VEC + k);
            acc[r] = fmaf(f[k], x.x, acc[r]); acc[r] = fmaf(f[k + 1], x.y, acc[r]); acc[r] = fmaf(f[k + 2], x.z, acc[r]); acc[r] = fmaf(f[k + 3], x.w, acc[r]);
          }
        }
    }
#pragma unroll
    for (int r = 0; r < LC_ROWS; r++) {
      const float v = warp_sum(acc[r]);
      if (lane == 0 && r < nr) a.out[(size_t)(r0 + r) * a.ldo + (size_t)h * a.vd + j] = from_f32<T>(v);
    }
  }
}

// The same for up to 16 rows on the tensor cores: the merged latents [16][rank], rounded to bf16, x W_uv of `LCM_OUT` values.
constexpr int LCM_ROWS = 16, LCM_OUT = 64, LCM_THREADS = 256;
static constexpr size_t lcm_smem(int rp) { return (size_t)2 * (LCM_ROWS + LCM_OUT) * (rp + 8); }

__global__ void __launch_bounds__(LCM_THREADS) latent_combine_mma_kernel(const LatentArgs<bf16> a, int R, int rp) {
  extern __shared__ __align__(16) unsigned char smem[];
  bf16 *sW = reinterpret_cast<bf16*>(smem), *sO = sW + (size_t)LCM_OUT * (rp + 8);  // rp: rank rounded up to 16
  __shared__ float wgt[LCM_ROWS][LS_MAX_NS];
  __shared__ int active[LCM_ROWS];
  __shared__ float red[4][2][32][4];
  const int h = blockIdx.x, j0 = blockIdx.y * LCM_OUT, r0 = blockIdx.z * LCM_ROWS, nr = min(LCM_ROWS, R - r0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  pdl_launch();
  for (int j = warp; j < LCM_OUT; j += LCM_THREADS / 32)  // parameters: ahead of the dependency wait
    for (int c = lane * 8; c < rp; c += 256) {
      bf16* dst = sW + (size_t)j * (rp + 8) + c;
      if (j0 + j < a.vd && c < a.ldu) cp16(dst, a.uv + ((size_t)h * a.vd + j0 + j) * a.ldu + c);
      else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
  cp_commit();
  pdl_wait();
  for (int r = warp; r < nr; r += LCM_THREADS / 32) {
    const int p = a.position(r0 + r), n = a.window > 0 ? min(p + 1, a.window) : p + 1, chunk = a.slice(n), na = (n + chunk - 1) / chunk;
    const float2 st = lane < na ? a.stat[((size_t)(r0 + r) * a.H + h) * a.ns + lane] : make_float2(-INFINITY, 0.f);
    const float sink = a.sink[h], M = fmaxf(warp_max(st.x), sink), e = expf(st.x - M);
    const float L = warp_sum(st.y * e) + expf(sink - M);
    wgt[r][lane] = e / L;
    if (lane == 0) active[r] = na;
  }
  __syncthreads();
  for (int r = warp; r < LCM_ROWS; r += LCM_THREADS / 32) {
    const int na = r < nr ? active[r] : 0;
    const float* part = a.part + ((size_t)(r0 + min(r, nr - 1)) * a.H + h) * a.ns * a.lat4;
    for (int c0 = 0; c0 < rp; c0 += 512) {  // four pieces of a row per lane: their loads overlap
      float4 v[4];
#pragma unroll
      for (int k = 0; k < 4; k++) v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 2
      for (int s = 0; s < na; s++) {
        const float w = wgt[r][s];
#pragma unroll
        for (int k = 0; k < 4; k++) {
          const int c = c0 + k * 128 + lane * 4;
          if (c < a.lat4) {
            const float4 x = *reinterpret_cast<const float4*>(part + (size_t)s * a.lat4 + c);
            v[k].x = fmaf(x.x, w, v[k].x); v[k].y = fmaf(x.y, w, v[k].y); v[k].z = fmaf(x.z, w, v[k].z); v[k].w = fmaf(x.w, w, v[k].w);
          }
        }
      }
#pragma unroll
      for (int k = 0; k < 4; k++) {
        const int c = c0 + k * 128 + lane * 4;
        if (c < rp) *reinterpret_cast<uint2*>(sO + (size_t)r * (rp + 8) + c) = make_uint2(pack_bf16(v[k].x, v[k].y), pack_bf16(v[k].z, v[k].w));
      }
    }
  }
  cp_wait<0>();
  __syncthreads();
  // warps 0-3 take 16 values each over the first half of the latent, warps 4-7 over the second
  const int cg = warp & 3, half = warp >> 2, kh = (rp / 32) * 16, k0 = half ? kh : 0, k1 = half ? rp : kh;
  float acc[2][4] = {};
  for (int k = k0; k < k1; k += 16) {
    uint32_t o[4], w[4];
    ldsm4(o, sO + (size_t)(lane & 15) * (rp + 8) + k + (lane >> 4) * 8);
    ldsm4(w, sW + (size_t)(cg * 16 + (lane >> 4) * 8 + (lane & 7)) * (rp + 8) + k + ((lane >> 3) & 1) * 8);
    mma_bf16(acc[0], o, w[0], w[1]);
    mma_bf16(acc[1], o, w[2], w[3]);
  }
  if (half)
#pragma unroll
    for (int j = 0; j < 2; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) red[cg][j][lane][i] = acc[j][i];
  __syncthreads();
  if (half) return;
  const int g = lane >> 2, tq = lane & 3;
#pragma unroll
  for (int j = 0; j < 2; j++)
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int r = g + 8 * (i >> 1), c = j0 + cg * 16 + j * 8 + tq * 2 + (i & 1);
      if (r < nr && c < a.vd) a.out[(size_t)(r0 + r) * a.ldo + (size_t)h * a.vd + c] = __float2bfloat16_rn(acc[j][i] + red[cg][j][lane][i]);
    }
}

// ------------------------------------------------------------------------------------------------ expanded form
// 64 consecutive tokens of a sequence x one head; warp w owns tokens 16 w .. 16 w + 15.
constexpr int LX_Q = 64, LX_KV = 64, LX_THREADS = 128;

template <int VT>  // value tiles of 8 columns, an even number
__global__ void __launch_bounds__(LX_THREADS) latent_chunk_kernel(const LatentArgs<bf16> a, int qkp) {
  extern __shared__ __align__(16) unsigned char smem[];
  const int ldq = qkp + 8, ldv = VT * 8 + 8;
  bf16* sQ = reinterpret_cast<bf16*>(smem);
  bf16* sK = sQ + (size_t)LX_Q * ldq;
  bf16* sV = sK + (size_t)2 * LX_KV * ldq;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, b = blockIdx.z;
  // the last tokens have the longest context: first
  const int q0 = (int)(gridDim.x - 1 - blockIdx.x) * LX_Q, nq = min(LX_Q, a.Sc - q0);
  pdl_wait();
  // keys 0 .. T_ctx - 1 are positions start - T_prev ..; token q0 + t is key T_prev + q0 + t
  const int own = a.T_prev + q0, last = own + nq - 1;
  const int first = a.window > 0 ? max(0, own - a.window + 1) : 0;
  const int kp = a.dim / 8, rp = a.rd / 8, pad = (qkp - a.qk()) / 8, vp = a.vd / 8, per = kp + rp + pad + VT;
  auto load_tile = [&](int base, int s) {
    bf16 *tk = sK + (size_t)s * LX_KV * ldq, *tv = sV + (size_t)s * LX_KV * ldv;
    int k = tid / per, c = tid % per;
    const int dk = LX_THREADS / per, dc = LX_THREADS % per;
    for (; k < LX_KV; k += dk, c += dc) {
      if (c >= per) { c -= per; k++; if (k >= LX_KV) break; }
      const size_t row = (size_t)b * a.T_ctx + base + k;
      const bool in = base + k <= last;
      bf16* d = c < kp + rp + pad ? tk + (size_t)k * ldq + c * 8 : tv + (size_t)k * ldv + (c - kp - rp - pad) * 8;
      if (!in || (c >= kp + rp && c < kp + rp + pad) || c >= kp + rp + pad + vp) { *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0); continue; }
      const bf16* src;
      if (c < kp) src = a.kv + row * a.ldkv + (size_t)h * a.dim + c * 8;
      else if (c < kp + rp) src = a.ctx + row * a.ldc + a.rank + (c - kp) * 8;
      else src = a.kv + row * a.ldkv + (size_t)a.H * a.dim + (size_t)h * a.vd + (c - kp - rp - pad) * 8;
      cp16(d, src);
    }
    cp_commit();
  };
  load_tile(first, 0);
  // queries: 16-byte pieces as they are, the first 2 * rot_pairs values behind the unrotated ones turned
  {
    const int qp = qkp / 8, turned = 2 * a.rot_pairs;
    for (int i = tid; i < LX_Q * qp; i += LX_THREADS) {
      const int t = i / qp, e = i % qp * 8;
      bf16* d = sQ + (size_t)t * ldq + e;
      if (t >= nq || e >= a.qk()) *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      else if (e < a.dim || e >= a.dim + turned) *reinterpret_cast<uint4*>(d) = ld_128(a.proj + ((size_t)(q0 + t) * a.B + b) * a.ldp + (size_t)h * a.qk() + e);
      else if (e + 8 > a.dim + turned) {  // a piece that turns in part
        for (int k = 0; k < 8; k++)
          if (e + k >= a.dim + turned) d[k] = a.proj[((size_t)(q0 + t) * a.B + b) * a.ldp + (size_t)h * a.qk() + e + k];
      }
    }
#pragma unroll 4
    for (int i = tid; i < nq * a.rot_pairs; i += LX_THREADS) {
      const int t = i / a.rot_pairs, k = i % a.rot_pairs;
      const bf16* q = a.proj + ((size_t)(q0 + t) * a.B + b) * a.ldp + (size_t)h * a.qk() + a.dim;
      const float2 cs = *reinterpret_cast<const float2*>(a.rot + ((size_t)(a.start + q0 + t) * a.rot_pairs + k) * 2);
      const float u = to_f32(q[k]), v = to_f32(q[k + a.rot_pairs]);
      bf16* d = sQ + (size_t)t * ldq + a.dim + k;
      d[0] = __float2bfloat16_rn(fmaf(u, cs.x, -v * cs.y));
      d[a.rot_pairs] = __float2bfloat16_rn(fmaf(v, cs.x, u * cs.y));
    }
  }
  float o[VT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < VT; j++)
#pragma unroll
    for (int i = 0; i < 4; i++) o[j][i] = 0.f;
  const int g = lane >> 2, tq = lane & 3;
  const int row0 = own + warp * 16 + g;  // key number of this thread's first token; the second is 8 further
  const float sl2 = a.scale * LOG2E;
  int s = 0;
  for (int base = first; base <= last; base += LX_KV, s ^= 1) {
    if (base + LX_KV <= last) { load_tile(base + LX_KV, s ^ 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    const bf16 *tk = sK + (size_t)s * LX_KV * ldq, *tv = sV + (size_t)s * LX_KV * ldv;
    float sc[8][4];
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) sc[j][i] = 0.f;
    for (int k = 0; k < qkp; k += 16) {
      uint32_t qf[4];
      ldsm4(qf, sQ + (size_t)(warp * 16 + (lane & 15)) * ldq + k + (lane >> 4) * 8);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        uint32_t kf[4];
        ldsm4(kf, tk + (size_t)(j * 8 + (lane >> 4) * 8 + (lane & 7)) * ldq + k + ((lane >> 3) & 1) * 8);
        mma_bf16(sc[j], qf, kf[0], kf[1]);
        mma_bf16(sc[j + 1], qf, kf[2], kf[3]);
      }
    }
    float mx[2] = {m[0], m[1]};
    const int w0 = own + warp * 16;  // this warp's tokens are keys w0 .. w0 + 15
    if (base + LX_KV - 1 <= w0 && (a.window <= 0 || w0 + 15 - base < a.window)) {  // every key of the tile is seen by all of them
#pragma unroll
      for (int j = 0; j < 8; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) {
          sc[j][i] *= sl2;
          mx[i >> 1] = fmaxf(mx[i >> 1], sc[j][i]);
        }
    } else {
#pragma unroll
      for (int j = 0; j < 8; j++)
#pragma unroll
        for (int i = 0; i < 4; i++) {
          const int back = row0 + 8 * (i >> 1) - (base + j * 8 + tq * 2 + (i & 1));
          sc[j][i] = (back >= 0 && (a.window <= 0 || back < a.window)) ? sc[j][i] * sl2 : -INFINITY;
          mx[i >> 1] = fmaxf(mx[i >> 1], sc[j][i]);
        }
    }
    float al[2], mu[2];
#pragma unroll
    for (int i = 0; i < 2; i++) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
      mu[i] = mx[i] == -INFINITY ? 0.f : mx[i];  // nothing seen yet: every weight below is exp2(-inf) = 0
      al[i] = ex2(m[i] - mu[i]);
      m[i] = mx[i];
      l[i] *= al[i];
    }
#pragma unroll
    for (int j = 0; j < VT; j++) { o[j][0] *= al[0]; o[j][1] *= al[0]; o[j][2] *= al[1]; o[j][3] *= al[1]; }
#pragma unroll
    for (int j = 0; j < 8; j++)
#pragma unroll
      for (int i = 0; i < 4; i++) {
        sc[j][i] = ex2(sc[j][i] - mu[i >> 1]);
        l[i >> 1] += sc[j][i];
      }
#pragma unroll
    for (int k = 0; k < 4; k++) {
      const uint32_t pf[4] = {pack_bf16(sc[2 * k][0], sc[2 * k][1]), pack_bf16(sc[2 * k][2], sc[2 * k][3]), pack_bf16(sc[2 * k + 1][0], sc[2 * k + 1][1]),
                              pack_bf16(sc[2 * k + 1][2], sc[2 * k + 1][3])};
#pragma unroll
      for (int j = 0; j < VT; j += 2) {
        uint32_t vf[4];
        ldsm4t(vf, tv + (size_t)(k * 16 + (lane & 15)) * ldv + j * 8 + (lane >> 4) * 8);
        mma_bf16(o[j], pf, vf[0], vf[1]);
        mma_bf16(o[j + 1], pf, vf[2], vf[3]);
      }
    }
    __syncthreads();
  }
  pdl_launch();
  const float sink = a.sink[h] * LOG2E;
#pragma unroll
  for (int i = 0; i < 2; i++) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    const float M = fmaxf(m[i], sink), e = exp2f(m[i] - M);
    l[i] = e / fmaf(l[i], e, exp2f(sink - M));
  }
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const int t = warp * 16 + g + 8 * i;
    if (t < nq) {
      bf16* dst = a.out + ((size_t)(q0 + t) * a.B + b) * a.ldo + (size_t)h * a.vd;
#pragma unroll
      for (int j = 0; j < VT; j++)
        if (j * 8 < a.vd) *reinterpret_cast<uint32_t*>(dst + j * 8 + tq * 2) = pack_bf16(o[j][2 * i] * l[i], o[j][2 * i + 1] * l[i]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ host side
static int round32(int n) { return (n + 31) & ~31; }
// tensor-core form of the absorbed path: heads per CTA / 16 (0: this shape stays on the CUDA cores)
static int mma_tiles(const jg_dev* dev, const jg_latent_desc* d, int* stages) {
  if (d->dtype != JG_BF16 || d->kv_rank > LS_MAX_RANK) return 0;
  const int lq = round32(d->kv_rank + d->rot_dim);
  const size_t limit = (size_t)dev->prop.sharedMemPerBlockOptin - 1024;
  const int mt = d->heads > 16 && d->kv_rank <= 512 ? 2 : 1;
  for (*stages = 2; *stages >= 1; (*stages)--)
    if ((mt == 2 ? lm_smem<2, 8>(lq, *stages) : lm_smem<1, 8>(lq, *stages)) <= limit) return mt;
  return 0;
}
constexpr int LATENT_MAX_PARTS = 32 * 160;  // (row, head, slice) triples of a call with few rows
static int latent_splits(const jg_dev* dev, const jg_latent_desc* d, int R, int heads_per_cta) {
  const long long span = d->window > 0 && d->window < d->rot_rows ? d->window : d->rot_rows;
  const int groups = (d->heads + heads_per_cta - 1) / heads_per_cta;
  long long ns = (heads_per_cta > 1 ? dev->sm_count : 2 * dev->sm_count) / ((long long)R * groups);
  if (ns > (span + 63) / 64) ns = (span + 63) / 64;
  if (ns > LATENT_MAX_PARTS / ((long long)R * d->heads)) ns = LATENT_MAX_PARTS / ((long long)R * d->heads);
  return ns < 1 ? 1 : (ns > LS_MAX_NS ? LS_MAX_NS : (int)ns);
}
// whether a portion of Sc tokens runs in expanded form (when the host knows where it starts)
constexpr int LATENT_MIN_EXPANDED = 16, LATENT_MAX_CTX = 16384;
static bool expandable(const jg_latent_desc* d, int Sc) {
  return d->dtype == JG_BF16 && Sc >= LATENT_MIN_EXPANDED && d->dim % 8 == 0 && d->rot_dim % 8 == 0 && d->vdim % 8 == 0 && d->kv_rank % 8 == 0 &&
         d->dim + d->rot_dim <= 256 && d->vdim <= 256;
}
static long long longest_ctx(const jg_latent_desc* d, int Sc) {
  long long prev = d->window > 0 ? (long long)d->window - 1 : d->rot_rows;
  if (prev + Sc > d->rot_rows) prev = d->rot_rows - Sc;
  if (prev < 0) prev = 0;
  return prev + Sc > LATENT_MAX_CTX ? LATENT_MAX_CTX : prev + Sc;
}

JG_API int jg_latent_scratch_bytes(const jg_latent_desc* d, int32_t B, int32_t Sc, uint64_t* out) {
  JG_REQUIRE(d != nullptr && out != nullptr && B > 0 && Sc > 0, "latent_scratch_bytes: bad arguments");
  uint64_t RH = (uint64_t)B * Sc * d->heads, wide = 0;
  if (expandable(d, Sc)) {
    wide = (uint64_t)B * longest_ctx(d, Sc) * 2 * (d->ldc + d->heads * (d->dim + d->vdim)) + 64;
    // longer contexts, and starts the host does not know, take the absorbed form in passes of this many rows
    const uint64_t few = (uint64_t)B * LATENT_MIN_EXPANDED * d->heads;
    if (RH > few) RH = few;
  }
  const uint64_t parts = RH > LATENT_MAX_PARTS ? RH : LATENT_MAX_PARTS;
  const uint64_t narrow = 4 * (RH * (uint64_t)round32(d->kv_rank + d->rot_dim) + parts * (uint64_t)(((d->kv_rank + 3) & ~3) + 2)) + 256;
  *out = narrow > wide ? narrow : wide;
  return JG_OK;
}

template <int MT, int NTW, int NW>
static int launch_mma(jg_dev* dev, const LatentArgs<bf16>& a, int R, int stages) {
  auto kern = latent_mma_kernel<MT, NTW, NW>;
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)dev->prop.sharedMemPerBlockOptin - 1024));
    set[dev->ordinal & 7] = true;
  }
  return jg_launch(dev, "latent_mma", kern, dim3((unsigned)a.ns, (unsigned)((a.H + 16 * MT - 1) / (16 * MT)), (unsigned)R), dim3(32 * NW), lm_smem<MT, NW>(a.lq, stages), a, stages);
}
template <int MT>
static int launch_mma_cols(jg_dev* dev, const LatentArgs<bf16>& a, int R, int stages) {
  if (a.rank <= 128) return launch_mma<MT, 2, 8>(dev, a, R, stages);
  const bool wide = lm_smem<MT, 16>(a.lq, stages) <= (size_t)dev->prop.sharedMemPerBlockOptin - 1024;
  if (a.rank <= 256) return wide ? launch_mma<MT, 2, 16>(dev, a, R, stages) : launch_mma<MT, 4, 8>(dev, a, R, stages);
  if (a.rank <= 512) return wide ? launch_mma<MT, 4, 16>(dev, a, R, stages) : launch_mma<MT, 8, 8>(dev, a, R, stages);
  return launch_mma<1, 16, 8>(dev, a, R, stages);
}
static int launch_scores(jg_dev* dev, const LatentArgs<float>& a, int R, int, int) {
  return jg_launch(dev, "latent_split", latent_split_kernel<float>, dim3((unsigned)R, (unsigned)a.H, (unsigned)a.ns), dim3(LS_THREADS), (size_t)a.lat() * 4, a);
}
static int launch_scores(jg_dev* dev, const LatentArgs<bf16>& a, int R, int mt, int stages) {
  if (mt == 2) return launch_mma_cols<2>(dev, a, R, stages);
  if (mt == 1) return launch_mma_cols<1>(dev, a, R, stages);
  return jg_launch(dev, "latent_split", latent_split_kernel<bf16>, dim3((unsigned)R, (unsigned)a.H, (unsigned)a.ns), dim3(LS_THREADS), (size_t)a.lat() * 4, a);
}

template <typename T, int ROWS>
static int launch_pre(jg_dev* dev, const LatentArgs<T>& a, const jg_latent_desc* d, int R) {
  auto kern = latent_pre_kernel<T, ROWS>;
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 2048 * ROWS * 4));
    set[dev->ordinal & 7] = true;
  }
  const unsigned slices = (unsigned)((d->kv_rank + LP_COLS - 1) / LP_COLS);
  return jg_launch(dev, "latent_pre", kern, dim3(d->heads * slices + 1, (unsigned)((R + ROWS - 1) / ROWS)), dim3(256), (size_t)ROWS * d->dim * 4, a, R);
}

// Three rows and more in bf16: all three stages on the tensor cores; 1 = not this call.
static int launch_rows(jg_dev*, const LatentArgs<float>&, const jg_latent_desc*, int, int, int) { return 1; }
static int launch_rows(jg_dev* dev, const LatentArgs<bf16>& a0, const jg_latent_desc* d, int R, int mt, int stages) {
  const int dp = (d->dim + 15) & ~15, rp = (d->kv_rank + 15) & ~15;
  const size_t limit = (size_t)dev->prop.sharedMemPerBlockOptin - 8192;
  if (R < 3 || mt == 0 || lpm_smem(dp) > limit || lcm_smem(rp) > limit) return 1;
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    if (cudaFuncSetAttribute(latent_pre_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit) != cudaSuccess ||
        cudaFuncSetAttribute(latent_combine_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit) != cudaSuccess)
      return jg_cuda_fail(cudaGetLastError(), "latent_pre_mma attributes", __FILE__, __LINE__);
    set[dev->ordinal & 7] = true;
  }
  LatentArgs<bf16> a = a0;
  a.slice_round = 2 * LM_TILE;  // fewer slices to merge
  const unsigned slices = (unsigned)((d->kv_rank + LP_COLS - 1) / LP_COLS);
  int rc = jg_launch(dev, "latent_pre_mma", latent_pre_mma_kernel, dim3(d->heads * slices + LPM_ROWS / 4, (unsigned)((R + LPM_ROWS - 1) / LPM_ROWS)), dim3(LPM_THREADS), lpm_smem(dp), a, R, dp);
  if (rc) return rc;
  rc = launch_scores(dev, a, R, mt, stages);
  if (rc) return rc;
  return jg_launch(dev, "latent_combine_mma", latent_combine_mma_kernel, dim3((unsigned)d->heads, (unsigned)((d->vdim + LCM_OUT - 1) / LCM_OUT), (unsigned)((R + LCM_ROWS - 1) / LCM_ROWS)),
                   dim3(LCM_THREADS), lcm_smem(rp), a, R, rp);
}

template <typename T>
static int run_absorbed(jg_dev* dev, LatentArgs<T> a, const jg_latent_desc* d) {
  const int R = a.B * a.Sc;
  int stages = 1;
  const int mt = mma_tiles(dev, d, &stages);
  a.lq = round32(d->kv_rank + d->rot_dim);
  a.ns = latent_splits(dev, d, R, mt ? 16 * mt : 1);
  a.lat4 = (d->kv_rank + 3) & ~3;
  a.slice_round = mt ? LM_TILE : 1;
  a.qt = (T*)d->scratch;
  a.part = (float*)(d->scratch + 4ull * R * d->heads * a.lq);
  a.stat = (float2*)(a.part + (size_t)R * d->heads * a.ns * a.lat4);
  int rc = launch_rows(dev, a, d, R, mt, stages);
  if (rc != 1) return rc;
  rc = R == 1 ? launch_pre<T, 1>(dev, a, d, R) : (R <= 4 ? launch_pre<T, 4>(dev, a, d, R) : launch_pre<T, 8>(dev, a, d, R));
  if (rc) return rc;
  rc = launch_scores(dev, a, R, mt, stages);
  if (rc) return rc;
  const int rg = (R + LC_ROWS - 1) / LC_ROWS;
  int outs = 32;  // as many CTAs as fill the machine, no more: each of them merges the slices anew
  while (outs < d->vdim && (long long)rg * d->heads * ((d->vdim + 2 * outs - 1) / (2 * outs)) >= dev->sm_count) outs *= 2;
  return jg_launch(dev, "latent_combine", latent_combine_kernel<T>, dim3((unsigned)d->heads, (unsigned)((d->vdim + outs - 1) / outs), (unsigned)rg), dim3(256),
                   (size_t)LC_ROWS * ((d->ld_u + 3) & ~3) * 4, a, R, outs);
}

template <int VT>
static int launch_chunk(jg_dev* dev, const LatentArgs<bf16>& a, int qkp) {
  auto kern = latent_chunk_kernel<VT>;
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)dev->prop.sharedMemPerBlockOptin - 1024));
    set[dev->ordinal & 7] = true;
  }
  const size_t smem = (size_t)2 * ((LX_Q + 2 * LX_KV) * (qkp + 8) + 2 * LX_KV * (VT * 8 + 8));
  return jg_launch(dev, "latent_chunk", kern, dim3((unsigned)((a.Sc + LX_Q - 1) / LX_Q), (unsigned)a.H, (unsigned)a.B), dim3(LX_THREADS), smem, a, qkp);
}

static int run_expanded(jg_dev* dev, LatentArgs<bf16> a, const jg_latent_desc* d) {
  const int R = a.B * a.Sc, N = d->heads * (d->dim + d->vdim), W = a.B * a.T_prev;
  a.ctx = (bf16*)d->scratch;
  a.kv = a.ctx + (((size_t)a.B * a.T_ctx * d->ldc + 31) & ~(size_t)31);
  a.ldkv = N;
  int rc = jg_launch(dev, "latent_write", latent_write_kernel<bf16>, dim3((unsigned)((R + W + 7) / 8)), dim3(256), 0, a, R);
  if (rc) return rc;
  DenseCall c = {};
  c.dtype = JG_BF16; c.epilogue = JG_DENSE_STORE; c.M = a.B * a.T_ctx; c.N = N; c.K = d->kv_rank; c.x = a.ctx; c.ldx = d->ldc;
  c.w[0] = a.uk; c.ldw = d->ld_u; c.y = (void*)a.kv; c.ldy = N;
  rc = jg_dense_call(dev, c);
  if (rc) return rc;
  const int qkp = (d->dim + d->rot_dim + 15) & ~15;
  if (d->vdim <= 64) return launch_chunk<8>(dev, a, qkp);
  if (d->vdim <= 128) return launch_chunk<16>(dev, a, qkp);
  return launch_chunk<32>(dev, a, qkp);
}
static int run_expanded(jg_dev*, const LatentArgs<float>&, const jg_latent_desc*) { return JG_ENOTSUP; }

template <typename T>
static int latent_run(jg_dev* dev, const jg_batch* bt, const jg_latent_desc* d) {
  LatentArgs<T> a = {};
  a.proj = (const T*)d->proj; a.pool = (T*)d->pool; a.bt = (const int32_t*)d->block_table; a.rot = (const float*)d->rot;
  a.norm_w = (const float*)d->norm_w; a.sink = (const float*)d->sink;
  a.uk = (const T*)d->ukv; a.uv = a.uk + (size_t)d->heads * d->dim * d->ld_u; a.out = (T*)d->out;
  a.pos = (const int32_t*)bt->pos; a.seq = (const int32_t*)bt->seq;
  a.B = bt->B; a.Sc = bt->Sc; a.H = d->heads; a.dim = d->dim; a.rd = d->rot_dim; a.vd = d->vdim; a.rank = d->kv_rank; a.window = d->window;
  a.ldp = d->ldp; a.ldo = d->ldo; a.ldc = d->ldc; a.ldu = d->ld_u; a.page = d->page; a.pps = d->pages_per_slot;
  a.rot_pairs = d->rot_pairs; a.rot_rows = d->rot_rows; a.eps = d->eps; a.scale = d->scale; a.start = bt->start;
  while ((1 << a.page_shift) < d->page) a.page_shift++;
  if (expandable(d, bt->Sc) && bt->start >= 0) {
    JG_REQUIRE(bt->start + bt->Sc <= d->rot_rows, "latent_attn: positions %d .. %d are outside the tables", bt->start, bt->start + bt->Sc);
    a.T_prev = d->window > 0 && d->window - 1 < bt->start ? d->window - 1 : bt->start;
    a.T_ctx = a.T_prev + bt->Sc;
    if (a.T_ctx <= LATENT_MAX_CTX) return run_expanded(dev, a, d);
  }
  if (!expandable(d, bt->Sc)) return run_absorbed(dev, a, d);
  // absorbed form in passes of LATENT_MIN_EXPANDED tokens per sequence: rows of a pass are contiguous, positions shift
  JG_REQUIRE(bt->start >= 0, "latent_attn: a portion of %d tokens needs its start on the host", bt->Sc);
  for (int s = 0; s < bt->Sc; s += LATENT_MIN_EXPANDED) {
    LatentArgs<T> q = a;
    q.Sc = bt->Sc - s < LATENT_MIN_EXPANDED ? bt->Sc - s : LATENT_MIN_EXPANDED;
    q.shift = s;
    q.proj = a.proj + (size_t)s * a.B * a.ldp;
    q.out = a.out + (size_t)s * a.B * a.ldo;
    int rc = run_absorbed(dev, q, d);
    if (rc) return rc;
  }
  return JG_OK;
}

JG_API int jg_latent_attn(jg_dev* dev, const jg_batch* b, const jg_latent_desc* d) {
  JG_ENTER(dev);
  JG_REQUIRE(d != nullptr && b != nullptr && b->B > 0 && b->Sc > 0 && jg_aligned(b->pos, 4) && jg_aligned(b->seq, 4), "latent_attn: bad batch");
  JG_REQUIRE(d->dtype == JG_F32 || d->dtype == JG_BF16, "latent_attn: unknown element type %d", d->dtype);
  JG_REQUIRE(d->heads > 0 && d->heads <= 65535 && d->dim > 0 && d->rot_dim > 0 && d->vdim > 0 && d->kv_rank > 0 && d->window >= 0, "latent_attn: bad shape");
  JG_REQUIRE(d->dim <= 2048 && d->rot_dim <= 4096, "latent_attn: heads of %d + %d values are too large", d->dim, d->rot_dim);
  if (d->kv_rank > LS_MAX_RANK) { jg_set_error("latent_attn: latents of %d values (largest supported: %d)", d->kv_rank, LS_MAX_RANK); return JG_ENOTSUP; }
  JG_REQUIRE(d->rot_pairs >= 0 && 2 * d->rot_pairs <= d->rot_dim && d->rot_rows > 0, "latent_attn: bad rotary table");
  const int vec = d->dtype == JG_F32 ? 4 : 8;
  JG_REQUIRE(d->ldp >= d->heads * (d->dim + d->rot_dim) + d->kv_rank + d->rot_dim && d->ldo >= d->heads * d->vdim && d->ldc >= d->kv_rank + d->rot_dim && d->ld_u >= d->kv_rank &&
             d->ldc % vec == 0 && d->ld_u % vec == 0 && d->ldo % 2 == 0, "latent_attn: bad row strides");
  JG_REQUIRE(d->page > 0 && (d->page & (d->page - 1)) == 0 && d->pages_per_slot > 0, "latent_attn: page size must be a power of two");
  const long long span = d->window > 0 ? (long long)d->window - 1 + b->Sc : (long long)d->rot_rows, cap = (long long)d->page * d->pages_per_slot;
  JG_REQUIRE(cap >= span || cap >= d->rot_rows, "latent_attn: %lld cached positions do not hold a window of %d and %d new tokens", cap, d->window, b->Sc);
  JG_REQUIRE(d->proj && jg_aligned(d->pool, 16) && jg_aligned(d->block_table, 4) && jg_aligned(d->rot, 4) && d->norm_w && d->sink && jg_aligned(d->ukv, 16) && jg_aligned(d->scratch, 16) &&
             jg_aligned(d->out, 4), "latent_attn: null or misaligned pointer");
  uint64_t need = 0;
  int rc = jg_latent_scratch_bytes(d, b->B, b->Sc, &need);
  if (rc) return rc;
  JG_REQUIRE(d->scratch_bytes >= need, "latent_attn: scratch of %llu bytes, %llu needed", (unsigned long long)d->scratch_bytes, (unsigned long long)need);
  return d->dtype == JG_F32 ? latent_run<float>(dev, b, d) : latent_run<bf16>(dev, b, d);
}
