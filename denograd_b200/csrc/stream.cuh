// What the kernels of the layer-list models (hybrid.py: recurrent mixers, latent attention, grouped norms around every
// sublayer) share: element types, the batch of a call, and the step between two sublayers on the fp32 residual stream.
//
// Element type T of weights and activations is bf16 (serving) or float (everything in 32 bits).  Independent of T, the
// residual stream, norms, attention scores and weights, gates and recurrent state are fp32.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

typedef __nv_bfloat16 bf16;

template <typename T> struct Elem;
template <> struct Elem<float> {
  static constexpr int VEC = 4;  // elements of a 16-byte chunk
};
template <> struct Elem<bf16> {
  static constexpr int VEC = 8;
};

#ifdef __CUDACC__
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// a 16-byte chunk as floats
__device__ __forceinline__ void unpack_chunk(const uint4& v, float (&o)[4]) {
  o[0] = __uint_as_float(v.x); o[1] = __uint_as_float(v.y); o[2] = __uint_as_float(v.z); o[3] = __uint_as_float(v.w);
}
__device__ __forceinline__ void unpack_chunk(const uint4& v, float (&o)[8]) {
  o[0] = __uint_as_float(v.x << 16); o[1] = __uint_as_float(v.x & 0xFFFF0000u);
  o[2] = __uint_as_float(v.y << 16); o[3] = __uint_as_float(v.y & 0xFFFF0000u);
  o[4] = __uint_as_float(v.z << 16); o[5] = __uint_as_float(v.z & 0xFFFF0000u);
  o[6] = __uint_as_float(v.w << 16); o[7] = __uint_as_float(v.w & 0xFFFF0000u);
}

__device__ __forceinline__ float sigmoid_f32(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }  // division within 2 ulp; 0 below -87
__device__ __forceinline__ float silu_f32(float z) { return z * sigmoid_f32(z); }
// z / 2 (1 + tanh(y)) = z sigmoid(2 y) with y = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh_f32(float z) { return z * sigmoid_f32(1.5957691216057308f * fmaf(0.044715f * z * z, z, z)); }
__device__ __forceinline__ float log_sigmoid_f32(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float softplus_f32(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
// minGRU: candidate state of a pre-activation
__device__ __forceinline__ float mingru_candidate(float u) { return u >= 0.0f ? u + 0.5f : sigmoid_f32(u); }
// gate clamped from above, linear part from both sides: min(g, l) * sigmoid(alpha * min(g, l)) * (clamp(u, -l, l) + 1)
constexpr float GLU_ALPHA = 1.702f;
__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f32(GLU_ALPHA * g) * (u + 1.0f);
}
// (value, lowest index) key of an fp32 logit: an unsigned maximum picks the largest value, the smallest index among equals
__device__ __forceinline__ unsigned long long argmax_key_f32(float v, uint32_t idx) {
  const uint32_t u = __float_as_uint(v);
  const uint32_t k = (u & 0x80000000u) ? ~u : (u | 0x80000000u);
  return ((unsigned long long)k << 32) | (unsigned long long)(0xFFFFFFFFu - idx);
}
#endif

// ------------------------------------------------------------------------------------------------ between two sublayers
// x <- x + norm(y) * w_add (skipped when y is null), then h = norm(x) * w_norm (skipped when w_norm is null): the norm
// after one sublayer, the residual sum and the norm before the next one, on one row.  norm divides each of `groups` equal
// consecutive parts by its own sqrt(mean(part^2) + eps).  A sublayer that reads the stream itself takes h = x (`plain`).
struct StreamArgs {
  const float* x;       // [R][D] residual stream
  const float* y;       // [R][D] what the sublayer returned, or null
  const float* w_add;   // [D]
  float* x_out;         // [R][D] stream after the sum, or null
  const float* w_norm;  // [D]
  const int32_t* rows;  // row indirection into x and y, or null
  int D, groups;
  float eps;
  int plain;            // h = x, whatever w_norm is
};

static inline int stream_units(int groups, int warps) { return groups >= warps ? groups : (warps / groups) * groups; }
// floats of shared memory one row needs: the row, and two sets of partial sums
static inline size_t stream_smem_floats(int D, int groups, int warps) { return (size_t)((D + 3) & ~3) + 2 * (size_t)stream_units(groups, warps); }

#ifdef __CUDACC__
// One row, by the NT threads of a CTA.  `buf` holds D floats and `red` 2 * stream_units; the caller synchronises before
// reusing them.  store(i, v) receives the V normalised values from element i on.
template <int NT, int V, typename Store>
__device__ __forceinline__ void stream_row_v(const StreamArgs& a, size_t src, float* x_out_row, float* buf, float* red, Store store) {
  constexpr int W = NT / 32;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int gs = a.D / a.groups, P = a.groups >= W ? 1 : W / a.groups, units = a.groups * P;
  const int plen = ((gs + P - 1) / P + V - 1) / V * V;
  const float* xr = a.x + src * a.D;
  const float* yr = a.y ? a.y + src * a.D : nullptr;
  float* red2 = red + units;
  auto load = [](const float* p, float (&v)[V]) {
    if constexpr (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
    else v[0] = p[0];
  };
  auto put = [](float* p, const float (&v)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else p[0] = v[0];
  };
  auto rstd = [&](const float* s, int g) {
    float t = 0.f;
    for (int p = 0; p < P; p++) t += s[g * P + p];
    return 1.0f / sqrtf(t / (float)gs + a.eps);
  };
  for (int u = warp; u < units; u += W) {  // a thread meets the same elements again below: buf needs no barrier
    const int g = u / P, lo = g * gs + (u % P) * plen, hi = min((g + 1) * gs, lo + plen);
    float ss = 0.f;
    for (int i = lo + lane * V; i < hi; i += 32 * V) {
      float v[V];
      load((yr ? yr : xr) + i, v);
      put(buf + i, v);
#pragma unroll
      for (int k = 0; k < V; k++) ss = fmaf(v[k], v[k], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[u] = ss;
  }
  __syncthreads();
  if (yr) {
    for (int u = warp; u < units; u += W) {
      const int g = u / P, lo = g * gs + (u % P) * plen, hi = min((g + 1) * gs, lo + plen);
      const float r = rstd(red, g);
      float ss = 0.f;
      for (int i = lo + lane * V; i < hi; i += 32 * V) {
        float v[V], x[V], w[V];
        load(buf + i, v);
        load(xr + i, x);
        load(a.w_add + i, w);
#pragma unroll
        for (int k = 0; k < V; k++) { x[k] = fmaf(v[k] * r, w[k], x[k]); ss = fmaf(x[k], x[k], ss); }
        put(buf + i, x);
        if (x_out_row) put(x_out_row + i, x);
      }
      ss = warp_sum(ss);
      if (lane == 0) red2[u] = ss;
    }
    __syncthreads();
  }
  if (a.plain) {
    for (int u = warp; u < units; u += W) {
      const int g = u / P, lo = g * gs + (u % P) * plen, hi = min((g + 1) * gs, lo + plen);
      for (int i = lo + lane * V; i < hi; i += 32 * V) {
        float v[V];
        load(buf + i, v);
        store(i, v);
      }
    }
    return;
  }
  if (a.w_norm == nullptr) return;
  for (int u = warp; u < units; u += W) {
    const int g = u / P, lo = g * gs + (u % P) * plen, hi = min((g + 1) * gs, lo + plen);
    const float r = rstd(yr ? red2 : red, g);
    for (int i = lo + lane * V; i < hi; i += 32 * V) {
      float v[V], w[V];
      load(buf + i, v);
      load(a.w_norm + i, w);
#pragma unroll
      for (int k = 0; k < V; k++) v[k] = v[k] * r * w[k];
      store(i, v);
    }
  }
}
template <int NT, typename Store>
__device__ __forceinline__ void stream_row(const StreamArgs& a, size_t src, float* x_out_row, float* buf, float* red, Store store) {
  if ((a.D / a.groups) % 4 == 0) stream_row_v<NT, 4>(a, src, x_out_row, buf, red, store);
  else stream_row_v<NT, 1>(a, src, x_out_row, buf, red, store);
}

// ------------------------------------------------------------------------------------------------ after a linear recurrence
// One row of o / den / rms(group) * w * sigmoid(gate) * scale (jg_gated_norm) by the NT threads of a CTA; buf holds
// gated_smem_floats.  Everything comes in at once: the divided read-outs and the factors behind the norm go to shared memory,
// where the groups' sums are taken.  store(i, v) receives the V values from element i on.
template <typename T>
struct GatedArgs {
  const float *o, *den, *w;
  const T* gate;
  int H, vd, groups, ldp, vec;  // vec: rows and heads come in pieces of four
  float eps, scale;
};
template <int NT, int V, typename T, typename Store>
__device__ __forceinline__ void gated_row_v(const GatedArgs<T>& a, size_t r, float* buf, Store store) {
  constexpr int W = NT / 32;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n = a.H * a.vd, n4 = (n + 3) & ~3;
  const int gs = n / a.groups, P = a.groups >= W ? 1 : W / a.groups, units = a.groups * P, plen = ((gs + P - 1) / P + V - 1) / V * V;
  const float *o = a.o + r * n, *den = a.den ? a.den + r * a.H : nullptr;
  const T* gate = a.gate + r * a.ldp;
  float *fac = buf + n4, *red = fac + n4;
#pragma unroll 4
  for (int i = threadIdx.x * V; i < n; i += NT * V) {
    const float d = den ? den[i / a.vd] : 1.f;
    if constexpr (V == 4) {
      float4 x = *reinterpret_cast<const float4*>(o + i), w = *reinterpret_cast<const float4*>(a.w + i);
      float g[4];
      if constexpr (sizeof(T) == 2) {
        const uint2 t = *reinterpret_cast<const uint2*>(gate + i);
        g[0] = __uint_as_float(t.x << 16); g[1] = __uint_as_float(t.x & 0xFFFF0000u); g[2] = __uint_as_float(t.y << 16); g[3] = __uint_as_float(t.y & 0xFFFF0000u);
      } else {
        const float4 t = *reinterpret_cast<const float4*>(gate + i);
        g[0] = t.x; g[1] = t.y; g[2] = t.z; g[3] = t.w;
      }
      if (den) { x.x /= d; x.y /= d; x.z /= d; x.w /= d; }
      w.x *= sigmoid_f32(g[0]); w.y *= sigmoid_f32(g[1]); w.z *= sigmoid_f32(g[2]); w.w *= sigmoid_f32(g[3]);
      *reinterpret_cast<float4*>(buf + i) = x;
      *reinterpret_cast<float4*>(fac + i) = w;
    } else {
      buf[i] = den ? o[i] / d : o[i];
      fac[i] = a.w[i] * sigmoid_f32(to_f32(gate[i]));
    }
  }
  __syncthreads();
  for (int u = warp; u < units; u += W) {
    const int g = u / P, lo = g * gs + (u % P) * plen, hi = min((g + 1) * gs, lo + plen);
    float ss = 0.f;
    for (int i = lo + lane * V; i < hi; i += 32 * V)
#pragma unroll
      for (int k = 0; k < V; k++) ss = fmaf(buf[i + k], buf[i + k], ss);
    ss = warp_sum(ss);
    if (lane == 0) red[u] = ss;
  }
  __syncthreads();
  for (int u = warp; u < units; u += W) {
    const int g = u / P, lo = g * gs + (u % P) * plen, hi = min((g + 1) * gs, lo + plen);
    float t = 0.f;
    for (int p = 0; p < P; p++) t += red[g * P + p];
    const float rs = a.scale / sqrtf(t / (float)gs + a.eps);
    for (int i = lo + lane * V; i < hi; i += 32 * V) {
      float v[V];
#pragma unroll
      for (int k = 0; k < V; k++) v[k] = buf[i + k] * rs * fac[i + k];
      store(i, v);
    }
  }
}
template <int NT, typename T, typename Store>
__device__ __forceinline__ void gated_row(const GatedArgs<T>& a, size_t r, float* buf, Store store) {
  if (a.vec) gated_row_v<NT, 4>(a, r, buf, store);
  else gated_row_v<NT, 1>(a, r, buf, store);
}
#endif
