// Attention over a sliding window and the sequence's first tokens (jg_window_desc): grouped heads, queries and keys normed over
// the whole projection, rotary positions on part of a head, keys and values in a paged ring whose first pages stay.
//
//   window_write    keys and values of new tokens into the cache (norm, rotation); prompt portions: queries into scratch
//   window_mma      bf16, one token or short portions: a context slice of one row for up to 16 heads of a kv head; every
//                   warp runs through its own tiles of 16 positions.  One token: it writes the cache row itself
//   window_split    the same for one head on the CUDA cores (fp32, and sizes the other does not take)
//   window_combine  context slices -> output
//   window_chunk    bf16 prompt portions: 64 or 128 queries of a head against tiles of 64 keys, one pass
//
// What a row sees is two runs of positions, the kept first ones and the window; both are numbered through (`Seen`), so tiles and
// slices go over one index.  Scores, softmax statistics and weights are fp32; on the tensor cores the weights meet the
// values in bf16.
#include <math.h>
#include <stddef.h>

#include "mma.cuh"

template <typename T>
struct WinArgs {
  const T *q, *k, *v;
  const float *qn, *kn, *rot;
  T* pool;
  const int32_t* bt;
  T* qs;         // portions: normed, rotated queries [R][H][dk8]
  float* part;   // [R][H][ns][vd4] weighted values of the slices
  float2* stat;  // [R][H][ns] their maxima and sums
  T* out;
  const int32_t *pos, *seq;
  int B, Sc, H, G, dim, vd, window, keep, ldp, ldo, page, page_shift, pps, pinned, pairs, rot_rows, dk8, dv8, vd4, ns, slice_round;
  float eps, scale, out_scale;
  __host__ __device__ __forceinline__ int row_size() const { return G * (dk8 + dv8); }
  // cache row of position p of the slot whose block-table row is `t`: its number, and where it is
  __device__ __forceinline__ uint32_t row_number(const int32_t* t, int p) const {
    const int i = p >> page_shift;
    return (uint32_t)t[i < pinned ? i : pinned + (i - pinned) % (pps - pinned)] * (uint32_t)page + (uint32_t)(p & (page - 1));
  }
  __device__ __forceinline__ T* row(const int32_t* t, int p) const { return pool + (size_t)row_number(t, p) * row_size(); }
  __device__ __forceinline__ int position(int r) const { return min(max(pos[r % B] + r / B, 0), rot_rows - 1); }
  __device__ __forceinline__ int slice(int n) const { return ((n + ns - 1) / ns + slice_round - 1) / slice_round * slice_round; }
};

// Positions that some row in [p0, p1] sees: the kept ones ahead of the window of p0, and from there to p1.
struct Seen {
  int kept, lo, n;
  __device__ __forceinline__ Seen(int p0, int p1, int window, int keep) {
    lo = window > 0 ? max(0, p0 - window + 1) : 0;
    kept = min(keep, lo);
    n = kept + p1 + 1 - lo;
  }
  __device__ __forceinline__ int at(int i) const { return i < kept ? i : lo + i - kept; }
};

template <int NT>
__device__ __forceinline__ float block_sum(float v, float* red) {  // red: NT / 32 floats, not in use
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; w++) s += red[w];
  return s;
}
template <typename T>
__device__ __forceinline__ float sum_squares(const T* x, int n, int tid, int nt) {
  float ss = 0.f;
  if (((uintptr_t)x & 15) == 0) {
    constexpr int V = Elem<T>::VEC;
    for (int i = tid; i < n / V; i += nt) {
      float f[V];
      unpack_chunk(ld_128(x + (size_t)i * V), f);
#pragma unroll
      for (int k = 0; k < V; k++) ss = fmaf(f[k], f[k], ss);
    }
    for (int i = n / V * V + tid; i < n; i += nt) { const float f = to_f32(x[i]); ss = fmaf(f, f, ss); }
  } else {
    for (int i = tid; i < n; i += nt) { const float f = to_f32(x[i]); ss = fmaf(f, f, ss); }
  }
  return ss;
}
// entry e of a normed and rotated head: x, w point at the head
template <typename T>
__device__ __forceinline__ float normed_rotated(const T* x, const float* w, float rs, int e, const float* cs, int pairs) {
  const float u = to_f32(x[e]) * rs * w[e];
  if (e >= 2 * pairs) return u;
  const int j = e < pairs ? e : e - pairs, p = e < pairs ? e + pairs : j;
  const float v = to_f32(x[p]) * rs * w[p], c = cs[2 * j], s = cs[2 * j + 1];
  return e < pairs ? fmaf(u, c, -v * s) : fmaf(u, c, v * s);
}

// `heads` heads of a row, normed and rotated, as T [heads][dk8] by NT threads.  Where heads and rotated pairs come in pieces of
// eight, a thread takes a piece and the one it turns with.
template <typename T, int NT>
__device__ __forceinline__ void write_heads(const WinArgs<T>& a, const T* x, const float* w, int heads, float rs, const float* cs, T* dst) {
  const int tid = threadIdx.x;
  if constexpr (sizeof(T) == 2) {
    if (a.dim % 8 == 0 && a.pairs % 8 == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)w & 15) == 0 && ((uintptr_t)cs & 15) == 0) {
      const int turned = a.pairs / 8, per = turned + (a.dim - 2 * a.pairs) / 8;
      auto piece = [&](int at, float (&v)[8]) {
        float f[8];
        unpack_chunk(ld_128(x + at), f);
        const float4 w0 = *reinterpret_cast<const float4*>(w + at), w1 = *reinterpret_cast<const float4*>(w + at + 4);
        v[0] = f[0] * rs * w0.x; v[1] = f[1] * rs * w0.y; v[2] = f[2] * rs * w0.z; v[3] = f[3] * rs * w0.w;
        v[4] = f[4] * rs * w1.x; v[5] = f[5] * rs * w1.y; v[6] = f[6] * rs * w1.z; v[7] = f[7] * rs * w1.w;
      };
      auto put = [&](int at, const float (&v)[8]) {
        *reinterpret_cast<uint4*>(dst + at) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
      };
      for (int i = tid; i < heads * per; i += NT) {
        const int h = i / per, c = i % per;
        float u[8], v[8];
        if (c >= turned) {
          const int e = h * a.dim + 2 * a.pairs + (c - turned) * 8;
          piece(e, u);
          put(e, u);
          continue;
        }
        const int e = h * a.dim + c * 8;
        piece(e, u);
        piece(e + a.pairs, v);
#pragma unroll
        for (int k = 0; k < 8; k += 2) {
          const float4 r = *reinterpret_cast<const float4*>(cs + (c * 8 + k) * 2);
          const float u0 = u[k], u1 = u[k + 1], v0 = v[k], v1 = v[k + 1];
          u[k] = fmaf(u0, r.x, -v0 * r.y); v[k] = fmaf(v0, r.x, u0 * r.y);
          u[k + 1] = fmaf(u1, r.z, -v1 * r.w); v[k + 1] = fmaf(v1, r.z, u1 * r.w);
        }
        put(e, u);
        put(e + a.pairs, v);
      }
      return;
    }
  }
  for (int i = tid; i < heads * a.dk8; i += NT) {
    const int h = i / a.dk8, e = i % a.dk8;
    dst[i] = from_f32<T>(e < a.dim ? normed_rotated(x + h * a.dim, w + h * a.dim, rs, e, cs, a.pairs) : 0.f);
  }
}

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) window_write_kernel(const WinArgs<T> a, int with_q) {
  __shared__ float red[2][8];
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x, tid = threadIdx.x, p = a.pos[r % a.B] + r / a.B;
  if (p < 0 || p >= a.rot_rows) return;  // outside the tables: left alone
  const T *q = a.q + (size_t)r * a.ldp, *k = a.k + (size_t)r * a.ldp, *v = a.v + (size_t)r * a.ldp;
  float sk = warp_sum(sum_squares(k, a.G * a.dim, tid, 256)), sq = with_q ? warp_sum(sum_squares(q, a.H * a.dim, tid, 256)) : 0.f;
  if ((tid & 31) == 0) { red[0][tid >> 5] = sk; red[1][tid >> 5] = sq; }
  T *dst = a.row(a.bt + (size_t)a.seq[r % a.B] * a.pps, p), *dv = dst + a.G * a.dk8;
  if (a.vd % Elem<T>::VEC == 0 && ((uintptr_t)v & 15) == 0 && a.dv8 == a.vd) {
    for (int i = tid * Elem<T>::VEC; i < a.G * a.vd; i += 256 * Elem<T>::VEC) *reinterpret_cast<uint4*>(dv + i) = ld_128(v + i);
  } else {
    for (int i = tid; i < a.G * a.dv8; i += 256) {
      const int g = i / a.dv8, e = i % a.dv8;
      dv[i] = e < a.vd ? v[g * a.vd + e] : from_f32<T>(0.f);
    }
  }
  __syncthreads();
  sk = sq = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) { sk += red[0][w]; sq += red[1][w]; }
  const float* cs = a.rot + (size_t)p * a.pairs * 2;
  write_heads<T, 256>(a, k, a.kn, a.G, 1.0f / sqrtf(sk / (float)(a.G * a.dim) + a.eps), cs, dst);
  if (with_q) write_heads<T, 256>(a, q, a.qn, a.H, 1.0f / sqrtf(sq / (float)(a.H * a.dim) + a.eps), cs, a.qs + (size_t)r * a.H * a.dk8);
}

// ------------------------------------------------------------------------------------------------ few rows, CUDA cores
constexpr int WS_THREADS = 128, WS_TILE = 64, WS_MAX_VDIM = 1024, WIN_MAX_NS = 32;

template <typename T>
__global__ void __launch_bounds__(WS_THREADS) window_split_kernel(const WinArgs<T> a) {
  constexpr int NR = WS_MAX_VDIM / WS_THREADS;
  extern __shared__ float sq[];  // this head's query
  __shared__ float sc[WS_TILE], red[WS_THREADS / 32];
  __shared__ const T* rows[WS_TILE];
  pdl_launch();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int r = blockIdx.x, h = blockIdx.y, g = h / (a.H / a.G), p = a.position(r);
  const int32_t* bt = a.bt + (size_t)a.seq[r % a.B] * a.pps;
  const Seen seen(p, p, a.window, a.keep);
  const int chunk = a.slice(seen.n), t0 = blockIdx.z * chunk, t1 = min(seen.n, t0 + chunk);
  if (t0 >= t1) return;  // nobody reads an empty slice
  const T* q = a.q + (size_t)r * a.ldp;
  const float rq = 1.0f / sqrtf(block_sum<WS_THREADS>(sum_squares(q, a.H * a.dim, tid, WS_THREADS), red) / (float)(a.H * a.dim) + a.eps);
  for (int e = tid; e < a.dim; e += WS_THREADS) sq[e] = normed_rotated(q + h * a.dim, a.qn + h * a.dim, rq, e, a.rot + (size_t)p * a.pairs * 2, a.pairs);
  const size_t id = ((size_t)r * a.H + h) * a.ns + blockIdx.z;
  float acc[NR], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int k = 0; k < NR; k++) acc[k] = 0.f;
  for (int base = t0; base < t1; base += WS_TILE) {
    const int nt = min(WS_TILE, t1 - base);
    __syncthreads();
    if (tid < nt) rows[tid] = a.row(bt, seen.at(base + tid));
    __syncthreads();
    for (int t = warp; t < nt; t += WS_THREADS / 32) {
      const T* c = rows[t] + g * a.dk8;
      float d = 0.f;
      for (int i = lane; i < a.dim; i += 32) d = fmaf(sq[i], to_f32(c[i]), d);
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
      const T* c = rows[t] + a.G * a.dk8 + g * a.dv8;
#pragma unroll
      for (int k = 0; k < NR; k++)
        if (tid + k * WS_THREADS < a.vd) acc[k] = fmaf(e, to_f32(c[tid + k * WS_THREADS]), acc[k]);
    }
  }
  if (a.ns == 1) {
    const float f = a.out_scale / l;
#pragma unroll
    for (int k = 0; k < NR; k++)
      if (tid + k * WS_THREADS < a.vd) a.out[(size_t)r * a.ldo + h * a.vd + tid + k * WS_THREADS] = from_f32<T>(acc[k] * f);
    return;
  }
  if (tid == 0) a.stat[id] = make_float2(m, l);
#pragma unroll
  for (int k = 0; k < NR; k++)
    if (tid + k * WS_THREADS < a.vd) a.part[id * a.vd4 + tid + k * WS_THREADS] = acc[k];
}

// one CTA per (head, row)
template <typename T>
__global__ void __launch_bounds__(128) window_combine_kernel(const WinArgs<T> a) {
  __shared__ float wgt[WIN_MAX_NS];
  pdl_launch();
  pdl_wait();
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, p = a.position(r);
  const Seen seen(p, p, a.window, a.keep);
  const int chunk = a.slice(seen.n), na = (seen.n + chunk - 1) / chunk;
  const size_t id = ((size_t)r * a.H + h) * a.ns;
  if (tid < 32) {
    const float2 st = tid < na ? a.stat[id + tid] : make_float2(-INFINITY, 0.f);
    const float M = warp_max(st.x), e = expf(st.x - M), L = warp_sum(st.y * e);
    wgt[tid] = e * (a.out_scale / L);
  }
  __syncthreads();
  for (int c = tid; c < a.vd; c += 128) {
    float v = 0.f;
#pragma unroll 4
    for (int s = 0; s < na; s++) v = fmaf(a.part[(id + s) * a.vd4 + c], wgt[s], v);
    a.out[(size_t)r * a.ldo + h * a.vd + c] = from_f32<T>(v);
  }
}

// ------------------------------------------------------------------------------------------------ few rows, tensor cores
// One row, up to 16 heads of one kv head, one context slice.  A warp scores 16 positions for all heads, turns the scores into
// weights in its registers and multiplies them with the values; its tiles are its own, so nothing waits until the warps'
// results are put together at the end.  KS: 16-wide steps of a key; VT: 8-wide tiles of a value.
constexpr int WM_WARPS = 4, WM_POS = 16, WM_STAGES = 3, WM_THREADS = 32 * WM_WARPS;
template <int KS, int VT>
struct WinTile {
  bf16 k[WM_POS][KS * 16 + 8], v[WM_POS][VT * 8 + 8];
};
template <int KS, int VT>
struct WinShared {
  union {
    WinTile<KS, VT> t[WM_WARPS][WM_STAGES];
    float o[WM_WARPS][16][VT * 8 + 2];
  };
  bf16 q[16][KS * 16 + 8];
  float m[WM_WARPS][16], l[WM_WARPS][16], red[2][WM_WARPS];
};
using WinSmallest = WinShared<4, 8>;
using WinLargest = WinShared<16, 32>;
static_assert(sizeof(WinTile<4, 8>) % 16 == 0 && sizeof(WinTile<16, 32>) % 16 == 0 && offsetof(WinSmallest, q) % 16 == 0 && offsetof(WinLargest, q) % 16 == 0, "tile layout");

template <int KS, int VT>
__global__ void __launch_bounds__(WM_THREADS) window_mma_kernel(const WinArgs<bf16> a, int fresh) {
  using WinTileT = WinTile<KS, VT>;
  extern __shared__ __align__(16) unsigned char wm_smem[];
  WinShared<KS, VT>& sh = *reinterpret_cast<WinShared<KS, VT>*>(wm_smem);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const int per = a.H / a.G, zg = (per + 15) / 16, kv = blockIdx.y / zg, hb = kv * per + blockIdx.y % zg * 16, nh = min(16, kv * per + per - hb), r = blockIdx.z;
  if (a.dk8 < KS * 16)  // what lies past the head in a key (a value's columns past the head are never used)
    for (int i = tid; i < (int)(sizeof(sh.t) / 16); i += WM_THREADS) reinterpret_cast<uint4*>(sh.t)[i] = make_uint4(0, 0, 0, 0);
  for (int i = tid; i < (int)(sizeof(sh.q) / 16); i += WM_THREADS) reinterpret_cast<uint4*>(sh.q)[i] = make_uint4(0, 0, 0, 0);
  pdl_launch();
  pdl_wait();
  const int p = a.position(r);
  const int32_t* bt = a.bt + (size_t)a.seq[r % a.B] * a.pps;
  const Seen seen(p, p, a.window, a.keep);
  const int chunk = a.slice(seen.n), t0 = blockIdx.x * chunk, t1 = min(seen.n, t0 + chunk);
  if (t0 >= t1) return;  // nobody reads an empty slice
  const float* cs = a.rot + (size_t)p * a.pairs * 2;
  if (fresh && t1 == seen.n) {  // the new token's keys and values
    const bf16 *k = a.k + (size_t)r * a.ldp, *v = a.v + (size_t)r * a.ldp + kv * a.vd;
    const float rk = 1.0f / sqrtf(block_sum<WM_THREADS>(sum_squares(k, a.G * a.dim, tid, WM_THREADS), sh.red[0]) / (float)(a.G * a.dim) + a.eps);
    bf16* dst = a.row(bt, p);
    for (int e = tid; e < a.dk8; e += WM_THREADS)
      dst[kv * a.dk8 + e] = from_f32<bf16>(e < a.dim ? normed_rotated(k + kv * a.dim, a.kn + kv * a.dim, rk, e, cs, a.pairs) : 0.f);
    for (int e = tid; e < a.dv8; e += WM_THREADS) dst[a.G * a.dk8 + kv * a.dv8 + e] = e < a.vd ? v[e] : from_f32<bf16>(0.f);
  }
  const bf16* q = a.q + (size_t)r * a.ldp;
  const float rq = 1.0f / sqrtf(block_sum<WM_THREADS>(sum_squares(q, a.H * a.dim, tid, WM_THREADS), sh.red[1]) / (float)(a.H * a.dim) + a.eps);
  for (int i = tid; i < nh * a.dim; i += WM_THREADS) {
    const int n = i / a.dim, e = i % a.dim;
    sh.q[n][e] = from_f32<bf16>(normed_rotated(q + (hb + n) * a.dim, a.qn + (hb + n) * a.dim, rq, e, cs, a.pairs));
  }
  __syncthreads();  // queries and the new cache row are there
  // a lane brings the same 16-byte pieces of every position: where they are in a cache row and in a tile's row
  constexpr int NP = (2 * KS + VT + 31) / 32;
  const int pk = a.dk8 / 8, rs = a.row_size();
  int from[NP], to[NP], step[NP];
#pragma unroll
  for (int n = 0; n < NP; n++) {
    const int c = lane + 32 * n, vc = c - pk;
    from[n] = c < pk ? kv * a.dk8 + c * 8 : vc < a.dv8 / 8 ? a.G * a.dk8 + kv * a.dv8 + vc * 8 : -1;
    to[n] = c < pk ? c * 8 : (int)(offsetof(WinTileT, v) / sizeof(bf16)) + vc * 8;
    step[n] = c < pk ? KS * 16 + 8 : VT * 8 + 8;
  }
  auto load = [&](int i) {  // this warp's i-th tile
    const int base = t0 + (warp + i * WM_WARPS) * WM_POS;
    if (base < t1) {
      bf16* t = reinterpret_cast<bf16*>(&sh.t[warp][i % WM_STAGES]);
      const uint32_t mine = a.row_number(bt, seen.at(min(base + (lane & 15), t1 - 1)));
#pragma unroll
      for (int n = 0; n < WM_POS; n++) {
        const bf16* src = a.pool + (size_t)__shfl_sync(0xffffffffu, mine, n) * rs;
#pragma unroll
        for (int c = 0; c < NP; c++)
          if (from[c] >= 0) cp16(t + to[c] + n * step[c], src + from[c]);
      }
    }
    cp_commit();
  };
#pragma unroll
  for (int i = 0; i < WM_STAGES - 1; i++) load(i);
  uint32_t qf[KS][4];
#pragma unroll
  for (int k = 0; k < KS; k++) ldsm4(qf[k], &sh.q[lane & 15][k * 16 + (lane >> 4) * 8]);
  float o[VT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < VT; j++)
#pragma unroll
    for (int i = 0; i < 4; i++) o[j][i] = 0.f;
  const float sl2 = a.scale * LOG2E;
  for (int i = 0; t0 + (warp + i * WM_WARPS) * WM_POS < t1; i++) {
    const int base = t0 + (warp + i * WM_WARPS) * WM_POS;
    __syncwarp();  // every lane is done with the tile that is replaced
    load(i + WM_STAGES - 1);
    cp_wait<WM_STAGES - 1>();
    __syncwarp();
    const WinTile<KS, VT>& t = sh.t[warp][i % WM_STAGES];
    float sc[2][4] = {};
#pragma unroll
    for (int k = 0; k < KS; k++) {
      uint32_t kf[4];
      ldsm4(kf, &t.k[(lane >> 4) * 8 + (lane & 7)][k * 16 + ((lane >> 3) & 1) * 8]);
      mma_bf16(sc[0], qf[k], kf[0], kf[1]);
      mma_bf16(sc[1], qf[k], kf[2], kf[3]);
    }
    float mx[2] = {m[0], m[1]}, al[2];
#pragma unroll
    for (int j = 0; j < 2; j++)
#pragma unroll
      for (int k = 0; k < 4; k++) {
        sc[j][k] = base + j * 8 + tq * 2 + (k & 1) < t1 ? sc[j][k] * sl2 : -INFINITY;
        mx[k >> 1] = fmaxf(mx[k >> 1], sc[j][k]);
      }
#pragma unroll
    for (int k = 0; k < 2; k++) {  // a tile has at least one position, so the maximum is finite
      mx[k] = fmaxf(mx[k], __shfl_xor_sync(0xffffffffu, mx[k], 1));
      mx[k] = fmaxf(mx[k], __shfl_xor_sync(0xffffffffu, mx[k], 2));
      al[k] = ex2(m[k] - mx[k]);
      m[k] = mx[k];
      l[k] *= al[k];
    }
#pragma unroll
    for (int j = 0; j < VT; j++) { o[j][0] *= al[0]; o[j][1] *= al[0]; o[j][2] *= al[1]; o[j][3] *= al[1]; }
#pragma unroll
    for (int j = 0; j < 2; j++)
#pragma unroll
      for (int k = 0; k < 4; k++) {
        sc[j][k] = ex2(sc[j][k] - m[k >> 1]);
        l[k >> 1] += sc[j][k];
      }
    const uint32_t pf[4] = {pack_bf16(sc[0][0], sc[0][1]), pack_bf16(sc[0][2], sc[0][3]), pack_bf16(sc[1][0], sc[1][1]), pack_bf16(sc[1][2], sc[1][3])};
#pragma unroll
    for (int j = 0; j < VT; j += 2) {
      uint32_t vf[4];
      ldsm4t(vf, &t.v[lane & 15][j * 8 + (lane >> 4) * 8]);
      mma_bf16(o[j], pf, vf[0], vf[1]);
      mma_bf16(o[j + 1], pf, vf[2], vf[3]);
    }
  }
  cp_wait<0>();
  __syncthreads();  // the tiles' memory takes the warps' results
#pragma unroll
  for (int k = 0; k < 2; k++) {
    l[k] += __shfl_xor_sync(0xffffffffu, l[k], 1);
    l[k] += __shfl_xor_sync(0xffffffffu, l[k], 2);
    if (tq == 0) { sh.m[warp][g + 8 * k] = m[k]; sh.l[warp][g + 8 * k] = l[k]; }
#pragma unroll
    for (int j = 0; j < VT; j++) *reinterpret_cast<float2*>(&sh.o[warp][g + 8 * k][j * 8 + tq * 2]) = make_float2(o[j][2 * k], o[j][2 * k + 1]);
  }
  __syncthreads();
  for (int n = warp; n < nh; n += WM_WARPS) {
    float M = -INFINITY, L = 0.f, w[WM_WARPS];
#pragma unroll
    for (int k = 0; k < WM_WARPS; k++) M = fmaxf(M, sh.m[k][n]);
#pragma unroll
    for (int k = 0; k < WM_WARPS; k++) {
      w[k] = ex2(sh.m[k][n] - M);  // a warp without tiles: 0
      L = fmaf(sh.l[k][n], w[k], L);
    }
    const size_t id = ((size_t)r * a.H + hb + n) * a.ns + blockIdx.x;
    const float f = a.ns == 1 ? a.out_scale / L : 1.f;
    if (a.ns > 1 && lane == 0) a.stat[id] = make_float2(M / LOG2E, L);
    for (int c = lane; c < a.vd; c += 32) {
      float x = 0.f;
#pragma unroll
      for (int k = 0; k < WM_WARPS; k++) x = fmaf(sh.o[k][n][c], w[k], x);
      if (a.ns == 1) a.out[(size_t)r * a.ldo + (hb + n) * a.vd + c] = from_f32<bf16>(x * f);
      else a.part[id * a.vd4 + c] = x;
    }
  }
}

// ------------------------------------------------------------------------------------------------ prompt portions
constexpr int WX_KV = 64;
static constexpr size_t wx_smem(int nq, int qkp, int vt) { return (size_t)2 * ((nq + 2 * WX_KV) * (qkp + 8) + 2 * WX_KV * (vt * 8 + 8)); }

// NW * 16 queries of one head; tiles of 64 seen positions, two in shared memory.
template <int VT, int NW>
__global__ void __launch_bounds__(32 * NW, VT <= 16 ? (NW == 8 ? 2 : 3) : 1) window_chunk_kernel(const WinArgs<bf16> a, int qkp) {
  constexpr int NQ = 16 * NW, NT = 32 * NW;
  extern __shared__ __align__(16) unsigned char wx_raw[];
  const int ldq = qkp + 8;
  constexpr int ldv = VT * 8 + 8;
  bf16 *sQ = reinterpret_cast<bf16*>(wx_raw), *sK = sQ + (size_t)NQ * ldq, *sV = sK + (size_t)2 * WX_KV * ldq;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * NQ, h = blockIdx.y, kv = h / (a.H / a.G), b = blockIdx.z, nq = min(NQ, a.Sc - q0);  // long ones first
  const int pieces = a.dk8 / 8, vpieces = a.dv8 / 8, per = pieces + vpieces;
  for (int i = tid; i < (int)(wx_smem(NQ, qkp, VT) / 16); i += NT) reinterpret_cast<uint4*>(wx_raw)[i] = make_uint4(0, 0, 0, 0);  // padding and missing rows
  __syncthreads();
  pdl_wait();
  const int p0 = a.pos[b] + q0, p1 = p0 + nq - 1;
  if (p0 < 0 || p1 >= a.rot_rows) return;
  const int32_t* bt = a.bt + (size_t)a.seq[b] * a.pps;
  const Seen seen(p0, p1, a.window, a.keep);
  // a lane brings the same 16-byte pieces of every key: where they are in a cache row and in a tile's row
  const int rs = a.row_size();
  auto load_tile = [&](int base, int s) {
    bf16 *tk = sK + (size_t)s * WX_KV * ldq, *tv = sV + (size_t)s * WX_KV * ldv;
    const uint32_t r0 = a.row_number(bt, seen.at(min(base + lane, seen.n - 1))), r1 = a.row_number(bt, seen.at(min(base + 32 + lane, seen.n - 1)));
    for (int c = lane; c < ((per + 31) & ~31); c += 32) {
      const int vc = c - pieces;
      const bf16* from = a.pool + (c < pieces ? kv * a.dk8 + c * 8 : a.G * a.dk8 + kv * a.dv8 + vc * 8);
      bf16* to = c < pieces ? tk + (size_t)warp * ldq + c * 8 : tv + (size_t)warp * ldv + vc * 8;
      const int step = NW * (c < pieces ? ldq : ldv);
#pragma unroll
      for (int i = 0; i < WX_KV / NW; i++) {  // keys past the end repeat the last one; they are masked below
        const int n = warp + i * NW;
        const uint32_t r = __shfl_sync(0xffffffffu, n < 32 ? r0 : r1, n & 31);
        if (c < per) cp16(to + i * step, from + (size_t)r * rs);
      }
    }
    cp_commit();
  };
  for (int i = tid; i < nq * pieces; i += NT) {
    const int t = i / pieces, c = i % pieces * 8;
    cp16(sQ + (size_t)t * ldq + c, a.qs + (((size_t)(q0 + t) * a.B + b) * a.H + h) * a.dk8 + c);
  }
  load_tile(0, 0);
  float o[VT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < VT; j++)
#pragma unroll
    for (int i = 0; i < 4; i++) o[j][i] = 0.f;
  const int w0 = p0 + warp * 16, w1 = w0 + 15;  // this warp's tokens
  const float sl2 = a.scale * LOG2E;
  int s = 0;
  for (int base = 0; base < seen.n; base += WX_KV, s ^= 1) {
    if (base + WX_KV < seen.n) { load_tile(base + WX_KV, s ^ 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    const int first = seen.at(base), end = base + WX_KV - 1, last = seen.at(min(end, seen.n - 1));
    // positions first .. last (in one run, or across the gap): all later than this warp's tokens, or all ahead of their windows?
    const bool none = first > w1 || (a.window > 0 && first >= a.keep && last <= w0 - a.window);
    if (!none) {
      const bool all = end < seen.n && last <= w0 && (a.window <= 0 || first > w1 - a.window || last < a.keep);  // seen by all of them
#pragma unroll 1
      for (int half = 0; half < 2; half++) {  // 32 keys at a time: fewer scores in registers
        const bf16 *tk = sK + (size_t)(s * WX_KV + half * 32) * ldq, *tv = sV + (size_t)(s * WX_KV + half * 32) * ldv;
        float sc[4][4];
#pragma unroll
        for (int j = 0; j < 4; j++)
#pragma unroll
          for (int i = 0; i < 4; i++) sc[j][i] = 0.f;
#pragma unroll 4
        for (int k = 0; k < qkp; k += 16) {
          uint32_t qf[4], k0[4], k1[4];
          ldsm4(qf, sQ + (size_t)(warp * 16 + (lane & 15)) * ldq + k + (lane >> 4) * 8);
          ldsm4(k0, tk + (size_t)((lane >> 4) * 8 + (lane & 7)) * ldq + k + ((lane >> 3) & 1) * 8);
          ldsm4(k1, tk + (size_t)(16 + (lane >> 4) * 8 + (lane & 7)) * ldq + k + ((lane >> 3) & 1) * 8);
          mma_bf16(sc[0], qf, k0[0], k0[1]);
          mma_bf16(sc[1], qf, k0[2], k0[3]);
          mma_bf16(sc[2], qf, k1[0], k1[1]);
          mma_bf16(sc[3], qf, k1[2], k1[3]);
        }
        float mx[2] = {m[0], m[1]};
        if (all) {
#pragma unroll
          for (int j = 0; j < 4; j++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
              sc[j][i] *= sl2;
              mx[i >> 1] = fmaxf(mx[i >> 1], sc[j][i]);
            }
        } else {
#pragma unroll
          for (int j = 0; j < 4; j++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
              const int v = base + half * 32 + j * 8 + tq * 2 + (i & 1), key = seen.at(v), back = w0 + g + 8 * (i >> 1) - key;
              sc[j][i] = v < seen.n && back >= 0 && (a.window <= 0 || back < a.window || key < a.keep) ? sc[j][i] * sl2 : -INFINITY;
              mx[i >> 1] = fmaxf(mx[i >> 1], sc[j][i]);
            }
        }
        float mu[2];
#pragma unroll
        for (int i = 0; i < 2; i++) {
          mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
          mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
          mu[i] = mx[i] == -INFINITY ? 0.f : mx[i];  // nothing seen yet: every weight below is 0
        }
        if (__any_sync(0xffffffffu, mx[0] != m[0] || mx[1] != m[1])) {
          const float a0 = ex2(m[0] - mu[0]), a1 = ex2(m[1] - mu[1]);
          l[0] *= a0;
          l[1] *= a1;
          m[0] = mx[0];
          m[1] = mx[1];
#pragma unroll
          for (int j = 0; j < VT; j++) { o[j][0] *= a0; o[j][1] *= a0; o[j][2] *= a1; o[j][3] *= a1; }
        }
#pragma unroll
        for (int j = 0; j < 4; j++)
#pragma unroll
          for (int i = 0; i < 4; i++) {
            sc[j][i] = ex2(sc[j][i] - mu[i >> 1]);
            l[i >> 1] += sc[j][i];
          }
#pragma unroll
        for (int k = 0; k < 2; k++) {
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
      }
    }
    __syncthreads();
  }
  pdl_launch();
#pragma unroll
  for (int i = 0; i < 2; i++) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    const int t = warp * 16 + g + 8 * i;
    if (t >= nq) continue;
    const float f = a.out_scale / l[i];
    bf16* dst = a.out + ((size_t)(q0 + t) * a.B + b) * a.ldo + (size_t)h * a.vd;
#pragma unroll
    for (int j = 0; j < VT; j++) {
      const int c = j * 8 + tq * 2;
      if (a.vd % 2 == 0) {
        if (c < a.vd) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[j][2 * i] * f, o[j][2 * i + 1] * f);
      } else {
        if (c < a.vd) dst[c] = __float2bfloat16_rn(o[j][2 * i] * f);
        if (c + 1 < a.vd) dst[c + 1] = __float2bfloat16_rn(o[j][2 * i + 1] * f);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ host side
constexpr int WINDOW_MIN_CHUNK = 16, WINDOW_MAX_PARTS = 32 * 160;
static bool on_tensor_cores(const jg_window_desc* d) { return d->dtype == JG_BF16 && d->dim <= 256 && d->vdim <= 256; }
static bool in_chunks(const jg_window_desc* d, int Sc) { return on_tensor_cores(d) && Sc >= WINDOW_MIN_CHUNK; }
static int heads_per_cta(const jg_window_desc* d) { return on_tensor_cores(d) ? (d->heads / d->kv_heads < 16 ? d->heads / d->kv_heads : 16) : 1; }
static int window_splits(const jg_dev* dev, const jg_window_desc* d, int R) {
  long long span = d->window > 0 ? (long long)d->window + d->keep : d->rot_rows;
  if (span > d->rot_rows) span = d->rot_rows;
  const int per = d->heads / d->kv_heads, hpc = heads_per_cta(d), groups = d->kv_heads * ((per + hpc - 1) / hpc);
  long long ns = 2ll * dev->sm_count / ((long long)R * groups);
  if (ns > (span + 63) / 64) ns = (span + 63) / 64;
  if (ns > WINDOW_MAX_PARTS / ((long long)R * d->heads)) ns = WINDOW_MAX_PARTS / ((long long)R * d->heads);
  return ns < 1 ? 1 : (ns > WIN_MAX_NS ? WIN_MAX_NS : (int)ns);
}

JG_API int jg_window_scratch_bytes(const jg_window_desc* d, int32_t B, int32_t Sc, uint64_t* out) {
  JG_REQUIRE(d != nullptr && out != nullptr && B > 0 && Sc > 0, "window_scratch_bytes: bad arguments");
  const uint64_t q = in_chunks(d, Sc) ? 2ull * B * Sc * d->heads * ((d->dim + 7) & ~7) : 0;
  const uint64_t parts = (uint64_t)WINDOW_MAX_PARTS * (((d->vdim + 3) & ~3) + 2) * 4;  // also enough for every call with fewer tokens
  *out = (q > parts ? q : parts) + 64;
  return JG_OK;
}

template <int KS, int VT>
static int launch_mma(jg_dev* dev, const WinArgs<bf16>& a, int groups, int R, int fresh) {
  auto kern = window_mma_kernel<KS, VT>;
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(WinShared<KS, VT>)));
    set[dev->ordinal & 7] = true;
  }
  return jg_launch(dev, "window_mma", kern, dim3((unsigned)a.ns, (unsigned)groups, (unsigned)R), dim3(WM_THREADS), sizeof(WinShared<KS, VT>), a, fresh);
}
template <int KS>
static int launch_mma_v(jg_dev* dev, const WinArgs<bf16>& a, int groups, int R, int fresh) {
  if (a.vd <= 64) return launch_mma<KS, 8>(dev, a, groups, R, fresh);
  if (a.vd <= 128) return launch_mma<KS, 16>(dev, a, groups, R, fresh);
  return launch_mma<KS, 32>(dev, a, groups, R, fresh);
}
template <int VT, int NW>
static int launch_wx(jg_dev* dev, const WinArgs<bf16>& a, int qkp) {
  auto kern = window_chunk_kernel<VT, NW>;
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)dev->prop.sharedMemPerBlockOptin - 1024));
    set[dev->ordinal & 7] = true;
  }
  return jg_launch(dev, "window_chunk", kern, dim3((unsigned)((a.Sc + 16 * NW - 1) / (16 * NW)), (unsigned)a.H, (unsigned)a.B), dim3(32 * NW), wx_smem(16 * NW, qkp, VT), a, qkp);
}
template <int VT>
static int launch_wx_rows(jg_dev* dev, const WinArgs<bf16>& a, int qkp) {
  // 128 queries per CTA when that still fills the machine and the shared memory holds it
  if ((long long)((a.Sc + 127) / 128) * a.H * a.B >= dev->sm_count && wx_smem(128, qkp, VT) <= dev->prop.sharedMemPerBlockOptin - 1024) return launch_wx<VT, 8>(dev, a, qkp);
  return launch_wx<VT, 4>(dev, a, qkp);
}

static int run_chunks(jg_dev*, const WinArgs<float>&) { return JG_ENOTSUP; }
static int run_chunks(jg_dev* dev, const WinArgs<bf16>& a) {
  int rc = jg_launch(dev, "window_write", window_write_kernel<bf16>, dim3((unsigned)(a.B * a.Sc)), dim3(256), 0, a, 1);
  if (rc) return rc;
  const int qkp = (a.dim + 15) & ~15;
  if (a.vd <= 64) return launch_wx_rows<8>(dev, a, qkp);
  if (a.vd <= 128) return launch_wx_rows<16>(dev, a, qkp);
  return launch_wx_rows<32>(dev, a, qkp);
}
static int run_mma(jg_dev*, const WinArgs<float>&, int, int) { return JG_ENOTSUP; }
static int run_mma(jg_dev* dev, const WinArgs<bf16>& a, int R, int fresh) {
  const int per = a.H / a.G, groups = a.G * ((per + 15) / 16);
  if (a.dim <= 64) return launch_mma_v<4>(dev, a, groups, R, fresh);
  if (a.dim <= 128) return launch_mma_v<8>(dev, a, groups, R, fresh);
  return launch_mma_v<16>(dev, a, groups, R, fresh);
}

template <typename T>
static int window_run(jg_dev* dev, const jg_batch* b, const jg_window_desc* d) {
  WinArgs<T> a = {};
  a.q = (const T*)d->q; a.k = (const T*)d->k; a.v = (const T*)d->v; a.qn = (const float*)d->q_norm; a.kn = (const float*)d->k_norm;
  a.rot = (const float*)d->rot; a.pool = (T*)d->pool; a.bt = (const int32_t*)d->block_table; a.out = (T*)d->out;
  a.pos = (const int32_t*)b->pos; a.seq = (const int32_t*)b->seq;
  a.B = b->B; a.Sc = b->Sc; a.H = d->heads; a.G = d->kv_heads; a.dim = d->dim; a.vd = d->vdim; a.window = d->window; a.keep = d->keep;
  a.ldp = d->ldp; a.ldo = d->ldo; a.page = d->page; a.pps = d->pages_per_slot; a.pinned = d->pinned; a.pairs = d->rot_pairs; a.rot_rows = d->rot_rows;
  a.eps = d->eps; a.scale = d->scale; a.out_scale = d->out_scale;
  a.dk8 = (d->dim + 7) & ~7; a.dv8 = (d->vdim + 7) & ~7; a.vd4 = (d->vdim + 3) & ~3;
  while ((1 << a.page_shift) < d->page) a.page_shift++;
  const int R = b->B * b->Sc;
  a.qs = (T*)d->scratch;
  if (in_chunks(d, b->Sc)) return run_chunks(dev, a);
  const bool mma = on_tensor_cores(d);
  a.ns = window_splits(dev, d, R);
  a.slice_round = mma ? WM_WARPS * WM_POS : 1;
  a.part = (float*)d->scratch;
  a.stat = (float2*)(a.part + (size_t)R * d->heads * a.ns * a.vd4);
  // a CTA with all heads of a kv head writes the new cache row itself
  const bool fresh = mma && b->Sc == 1 && d->heads / d->kv_heads <= 16;
  int rc = JG_OK;
  if (!fresh) rc = jg_launch(dev, "window_write", window_write_kernel<T>, dim3((unsigned)R), dim3(256), 0, a, 0);
  if (rc) return rc;
  if (mma) rc = run_mma(dev, a, R, fresh);
  else rc = jg_launch(dev, "window_split", window_split_kernel<T>, dim3((unsigned)R, (unsigned)d->heads, (unsigned)a.ns), dim3(WS_THREADS), (size_t)d->dim * 4, a);
  if (rc || a.ns == 1) return rc;
  return jg_launch(dev, "window_combine", window_combine_kernel<T>, dim3((unsigned)d->heads, (unsigned)R), dim3(128), 0, a);
}

JG_API int jg_window_attn(jg_dev* dev, const jg_batch* b, const jg_window_desc* d) {
  JG_ENTER(dev);
  JG_REQUIRE(d != nullptr && b != nullptr && b->B > 0 && b->Sc > 0 && jg_aligned(b->pos, 4) && jg_aligned(b->seq, 4), "window_attn: bad batch");
  JG_REQUIRE(d->dtype == JG_F32 || d->dtype == JG_BF16, "window_attn: unknown element type %d", d->dtype);
  JG_REQUIRE(d->heads > 0 && d->heads <= 65535 && d->kv_heads > 0 && d->heads % d->kv_heads == 0 && d->dim > 0 && d->vdim > 0 && d->window >= 0 && d->keep >= 0, "window_attn: bad shape");
  if (d->vdim > WS_MAX_VDIM || d->dim > 8192) { jg_set_error("window_attn: heads of %d / %d values (largest supported: 8192 / %d)", d->dim, d->vdim, WS_MAX_VDIM); return JG_ENOTSUP; }
  JG_REQUIRE(d->rot_pairs >= 0 && 2 * d->rot_pairs <= d->dim && d->rot_rows > 0, "window_attn: bad rotary table");
  JG_REQUIRE(d->ldp >= d->heads * d->dim && d->ldp >= d->kv_heads * d->vdim && d->ldo >= d->heads * d->vdim && d->ldo % 2 == 0, "window_attn: bad row strides");
  JG_REQUIRE(d->page > 0 && (d->page & (d->page - 1)) == 0 && d->pinned >= 0 && d->pages_per_slot > d->pinned, "window_attn: bad pages");
  // pinned pages hold the kept tokens; the others the window and the new tokens; or all positions have a page of their own
  const long long ring = (long long)d->page * (d->pages_per_slot - d->pinned), all = (long long)d->page * d->pages_per_slot;
  JG_REQUIRE(all >= d->rot_rows || (d->window > 0 && (long long)d->pinned * d->page >= d->keep && ring >= (long long)d->window - 1 + b->Sc),
             "window_attn: the cache does not hold a window of %d, %d first tokens and %d new ones", d->window, d->keep, b->Sc);
  JG_REQUIRE(d->q && d->k && d->v && jg_aligned(d->q_norm, 4) && jg_aligned(d->k_norm, 4) && jg_aligned(d->rot, 4) && jg_aligned(d->pool, 16) && jg_aligned(d->block_table, 4) &&
             jg_aligned(d->scratch, 16) && jg_aligned(d->out, 4), "window_attn: null or misaligned pointer");
  uint64_t need = 0;
  int rc = jg_window_scratch_bytes(d, b->B, b->Sc, &need);
  if (rc) return rc;
  JG_REQUIRE(d->scratch_bytes >= need, "window_attn: scratch of %llu bytes, %llu needed", (unsigned long long)d->scratch_bytes, (unsigned long long)need);
  return d->dtype == JG_F32 ? window_run<float>(dev, b, d) : window_run<bf16>(dev, b, d);
}
