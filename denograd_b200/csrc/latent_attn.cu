// Latent attention over a paged ring of (normed latent | rotated key part) rows: a sliding window, a learned sink in the
// softmax's denominator, YaRN-scaled half-split rotary on the shared key part.
//
//   latent_write    per row: RMS norm of the latent, rotation of the key part, cache row
//   decode, short portions, fp32 ("absorbed"): the per-head key and value projections are applied to the query and to
//                   the attended latent instead of to every cached position —
//                   latent_absorb   qt = [W_uk^T q_unrotated | rotated q]
//                   latent_split    scores qt . cache row, softmax statistics and the weighted latent of a context slice
//                   latent_combine  slices + sink -> latent, then W_uv
//
// Scores, softmax statistics and weights are fp32.
#include <math.h>
#include <stdlib.h>

#include "dense.cuh"

template <typename T>
struct LatentArgs {
  const T* proj;
  T* pool;
  const int32_t* bt;
  const float *rot, *norm_w, *sink;
  const T *uk, *uv;
  float *qt, *part;
  T* out;
  const int32_t *pos, *seq;
  int B, Sc, H, dim, rd, vd, rank, window, ldp, ldo, ldc, ldu, page, page_shift, pps, rot_pairs, rot_rows, ns;
  float eps, scale;
  __device__ __forceinline__ int qk() const { return dim + rd; }
  __device__ __forceinline__ int lat() const { return rank + rd; }
  // cache row of position p of the slot whose block-table row is `t`
  __device__ __forceinline__ T* row(const int32_t* t, int p) const {
    return pool + ((size_t)t[(p >> page_shift) % pps] * page + (p & (page - 1))) * ldc;
  }
};

// Entry i of a rotated vector: pairs (i, i + rot_pairs) turn, the rest passes.
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int i, const float* cs, int pairs) {
  if (i >= 2 * pairs) return to_f32(x[i]);
  const int j = i < pairs ? i : i - pairs;
  const float u = to_f32(x[j]), v = to_f32(x[j + pairs]), c = cs[2 * j], s = cs[2 * j + 1];
  return i < pairs ? fmaf(u, c, -v * s) : fmaf(v, c, u * s);
}

template <typename T>
__global__ void __launch_bounds__(256) latent_write_kernel(const LatentArgs<T> a, int R) {
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= R) return;
  const int b = r % a.B, p = a.pos[b] + r / a.B;
  if (p < 0 || p >= a.rot_rows) return;  // outside the tables: left alone
  const T* c = a.proj + (size_t)r * a.ldp + a.H * a.qk();
  T* dst = a.row(a.bt + (size_t)a.seq[b] * a.pps, p);
  float ss = 0.f;
  for (int i = lane; i < a.rank; i += 32) { const float v = to_f32(c[i]); ss = fmaf(v, v, ss); }
  const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)a.rank + a.eps);
  for (int i = lane; i < a.rank; i += 32) dst[i] = from_f32<T>(to_f32(c[i]) * rs * a.norm_w[i]);
  const float* cs = a.rot + (size_t)p * a.rot_pairs * 2;
  for (int i = lane; i < a.rd; i += 32) dst[a.rank + i] = from_f32<T>(rotated(c + a.rank, i, cs, a.rot_pairs));
}

// ------------------------------------------------------------------------------------------------ absorbed form
template <typename T>
__global__ void __launch_bounds__(128) latent_absorb_kernel(const LatentArgs<T> a) {
  extern __shared__ float sq[];
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y, b = r % a.B, p = min(max(a.pos[b] + r / a.B, 0), a.rot_rows - 1);
  const T* q = a.proj + (size_t)r * a.ldp + (size_t)h * a.qk();
  for (int i = threadIdx.x; i < a.dim; i += 128) sq[i] = to_f32(q[i]);
  __syncthreads();
  float* qt = a.qt + ((size_t)r * a.H + h) * a.lat();
  const T* uk = a.uk + (size_t)h * a.dim * a.ldu;
  for (int i = threadIdx.x; i < a.rank; i += 128) {
    float acc = 0.f;
    for (int d = 0; d < a.dim; d++) acc = fmaf(sq[d], to_f32(uk[(size_t)d * a.ldu + i]), acc);
    qt[i] = acc;
  }
  const float* cs = a.rot + (size_t)p * a.rot_pairs * 2;
  for (int i = threadIdx.x; i < a.rd; i += 128) qt[a.rank + i] = rotated(q + a.dim, i, cs, a.rot_pairs);
}

constexpr int LS_THREADS = 128, LS_TILE = 64, LS_MAX_RANK = 1024;

template <typename T>
__global__ void __launch_bounds__(LS_THREADS) latent_split_kernel(const LatentArgs<T> a) {
  constexpr int NR = LS_MAX_RANK / LS_THREADS;
  extern __shared__ float sq[];  // qt of this (row, head)
  __shared__ float sc[LS_TILE];
  __shared__ const T* rows[LS_TILE];
  pdl_launch();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int r = blockIdx.x, h = blockIdx.y, b = r % a.B, p = min(max(a.pos[b] + r / a.B, 0), a.rot_rows - 1), L = a.lat();
  const int32_t* bt = a.bt + (size_t)a.seq[b] * a.pps;
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0, n = p + 1 - lo;
  const int chunk = (n + a.ns - 1) / a.ns, t0 = lo + blockIdx.z * chunk, t1 = min(p + 1, t0 + chunk);
  float* part = a.part + (((size_t)r * a.H + h) * a.ns + blockIdx.z) * (a.rank + 2);
  for (int i = tid; i < L; i += LS_THREADS) sq[i] = a.qt[((size_t)r * a.H + h) * L + i];
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
  if (tid == 0) { part[0] = m; part[1] = l; }
#pragma unroll
  for (int k = 0; k < NR; k++)
    if (tid + k * LS_THREADS < a.rank) part[2 + tid + k * LS_THREADS] = acc[k];
}

template <typename T>
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentArgs<T> a) {
  extern __shared__ float so[];  // the attended latent
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float* part = a.part + ((size_t)r * a.H + h) * a.ns * (a.rank + 2);
  float M = a.sink[h];
  for (int s = 0; s < a.ns; s++) M = fmaxf(M, part[(size_t)s * (a.rank + 2)]);
  float l = expf(a.sink[h] - M);
  for (int s = 0; s < a.ns; s++) l += part[(size_t)s * (a.rank + 2) + 1] * expf(part[(size_t)s * (a.rank + 2)] - M);
  const float rl = 1.0f / l;
  for (int i = threadIdx.x; i < a.rank; i += 128) {
    float v = 0.f;
    for (int s = 0; s < a.ns; s++) v = fmaf(part[(size_t)s * (a.rank + 2) + 2 + i], expf(part[(size_t)s * (a.rank + 2)] - M), v);
    so[i] = v * rl;
  }
  __syncthreads();
  for (int j = warp; j < a.vd; j += 4) {
    const T* w = a.uv + ((size_t)h * a.vd + j) * a.ldu;
    float d = 0.f;
    for (int i = lane; i < a.rank; i += 32) d = fmaf(to_f32(w[i]), so[i], d);
    d = warp_sum(d);
    if (lane == 0) a.out[(size_t)r * a.ldo + (size_t)h * a.vd + j] = from_f32<T>(d);
  }
}

// ------------------------------------------------------------------------------------------------ host side
constexpr int LS_MAX_PARTS = 296;  // two CTAs per SM
static int latent_splits(const jg_latent_desc* d, int R) {
  const long long span = d->window > 0 ? d->window : d->rot_rows;
  long long ns = LS_MAX_PARTS / ((long long)R * d->heads > 0 ? (long long)R * d->heads : 1);
  if (ns > (span + 63) / 64) ns = (span + 63) / 64;
  return ns < 1 ? 1 : (ns > 32 ? 32 : (int)ns);
}

JG_API int jg_latent_scratch_bytes(const jg_latent_desc* d, int32_t B, int32_t Sc, uint64_t* out) {
  JG_REQUIRE(d != nullptr && out != nullptr && B > 0 && Sc > 0, "latent_scratch_bytes: bad arguments");
  const uint64_t RH = (uint64_t)B * Sc * d->heads;
  // slices: one per (row, head), or up to LS_MAX_PARTS in all when there are fewer (any smaller call fits too)
  *out = 4 * (RH * (uint64_t)(d->kv_rank + d->rot_dim) + (RH > LS_MAX_PARTS ? RH : LS_MAX_PARTS) * (uint64_t)(d->kv_rank + 2)) + 256;
  return JG_OK;
}

template <typename T>
static int latent_run(jg_dev* dev, const jg_batch* bt, const jg_latent_desc* d) {
  LatentArgs<T> a = {};
  a.proj = (const T*)d->proj; a.pool = (T*)d->pool; a.bt = (const int32_t*)d->block_table; a.rot = (const float*)d->rot;
  a.norm_w = (const float*)d->norm_w; a.sink = (const float*)d->sink;
  a.uk = (const T*)d->ukv; a.uv = a.uk + (size_t)d->heads * d->dim * d->ld_u; a.out = (T*)d->out;
  a.pos = (const int32_t*)bt->pos; a.seq = (const int32_t*)bt->seq;
  a.B = bt->B; a.Sc = bt->Sc; a.H = d->heads; a.dim = d->dim; a.rd = d->rot_dim; a.vd = d->vdim; a.rank = d->kv_rank; a.window = d->window;
  a.ldp = d->ldp; a.ldo = d->ldo; a.ldc = d->ldc; a.ldu = d->ld_u; a.page = d->page; a.pps = d->pages_per_slot;
  a.rot_pairs = d->rot_pairs; a.rot_rows = d->rot_rows; a.eps = d->eps; a.scale = d->scale;
  while ((1 << a.page_shift) < d->page) a.page_shift++;
  const int R = bt->B * bt->Sc, L = d->kv_rank + d->rot_dim;
  a.ns = latent_splits(d, R);
  a.qt = (float*)d->scratch;
  a.part = a.qt + (size_t)R * d->heads * L;
  int rc = jg_launch(dev, "latent_write", latent_write_kernel<T>, dim3((unsigned)((R + 7) / 8)), dim3(256), 0, a, R);
  if (rc) return rc;
  rc = jg_launch(dev, "latent_absorb", latent_absorb_kernel<T>, dim3((unsigned)R, (unsigned)d->heads), dim3(128), (size_t)d->dim * 4, a);
  if (rc) return rc;
  rc = jg_launch(dev, "latent_split", latent_split_kernel<T>, dim3((unsigned)R, (unsigned)d->heads, (unsigned)a.ns), dim3(LS_THREADS), (size_t)L * 4, a);
  if (rc) return rc;
  return jg_launch(dev, "latent_combine", latent_combine_kernel<T>, dim3((unsigned)R, (unsigned)d->heads), dim3(128), (size_t)d->kv_rank * 4, a);
}

JG_API int jg_latent_attn(jg_dev* dev, const jg_batch* b, const jg_latent_desc* d) {
  JG_ENTER(dev);
  JG_REQUIRE(d != nullptr && b != nullptr && b->B > 0 && b->Sc > 0 && jg_aligned(b->pos, 4) && jg_aligned(b->seq, 4), "latent_attn: bad batch");
  JG_REQUIRE(d->dtype == JG_F32 || d->dtype == JG_BF16, "latent_attn: unknown element type %d", d->dtype);
  JG_REQUIRE(d->heads > 0 && d->heads <= 65535 && d->dim > 0 && d->rot_dim > 0 && d->vdim > 0 && d->kv_rank > 0 && d->window >= 0, "latent_attn: bad shape");
  JG_REQUIRE(d->dim <= 4096 && d->kv_rank + d->rot_dim <= 8192, "latent_attn: heads of %d or latents of %d values are too large", d->dim, d->kv_rank);
  if (d->kv_rank > LS_MAX_RANK) { jg_set_error("latent_attn: latents of %d values (largest supported: %d)", d->kv_rank, LS_MAX_RANK); return JG_ENOTSUP; }
  JG_REQUIRE(d->rot_pairs >= 0 && 2 * d->rot_pairs <= d->rot_dim && d->rot_rows > 0, "latent_attn: bad rotary table");
  JG_REQUIRE(d->ldp >= d->heads * (d->dim + d->rot_dim) + d->kv_rank + d->rot_dim && d->ldo >= d->heads * d->vdim && d->ldc >= d->kv_rank + d->rot_dim && d->ld_u >= d->kv_rank,
             "latent_attn: row strides too small");
  JG_REQUIRE(d->page > 0 && (d->page & (d->page - 1)) == 0 && d->pages_per_slot > 0, "latent_attn: page size must be a power of two");
  const long long span = d->window > 0 ? (long long)d->window - 1 + b->Sc : (long long)d->rot_rows, cap = (long long)d->page * d->pages_per_slot;
  JG_REQUIRE(cap >= span || cap >= d->rot_rows, "latent_attn: %lld cached positions do not hold a window of %d and %d new tokens", cap, d->window, b->Sc);
  JG_REQUIRE(d->proj && d->pool && jg_aligned(d->block_table, 4) && jg_aligned(d->rot, 4) && d->norm_w && d->sink && d->ukv && jg_aligned(d->scratch, 16) && d->out, "latent_attn: null pointer");
  uint64_t need = 0;
  int rc = jg_latent_scratch_bytes(d, b->B, b->Sc, &need);
  if (rc) return rc;
  JG_REQUIRE(d->scratch_bytes >= need, "latent_attn: scratch of %llu bytes, %llu needed", (unsigned long long)d->scratch_bytes, (unsigned long long)need);
  return d->dtype == JG_F32 ? latent_run<float>(dev, b, d) : latent_run<bf16>(dev, b, d);
}
