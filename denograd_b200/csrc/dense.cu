// Projections of the layer-list models: y = epilogue(x W^T + b) with T = bf16 or float operands and fp32 accumulation.
//
//   1-2 rows   weight-streaming matrix-vector kernel (the scheme of gemv.cu: warp-private runs of output rows, a
//              cooperative remainder, an L2 prefetch ahead of the dependency wait).  Its prologue can take the rows straight
//              from the fp32 residual stream — post-norm of the previous sublayer, residual sum and pre-norm (stream.cuh) —
//              so that a decode step has no launch of its own for them; every CTA recomputes the row, CTA 0 writes the
//              new stream to a second buffer.
//   more rows  bf16: tcgen05 kernel (dense_tc.cu); float: a register-tiled fp32 kernel (no reduced-precision modes).
//
// The prologue can also finish a linear recurrence (division, norm and output gate of jg_gated_norm).
//
// Epilogues: STORE (T or fp32; activation on some columns, some columns in fp32 elsewhere), GLU (clamped gate x linear, two matrices with biases), MINGRU (three matrices: update gate,
// candidate, output gate; advances the recurrence by one token and gates it), LOGITS (fp32 + argmax key).
#include "dense.cuh"

template <typename T>
struct MvArgs {
  const T* x;
  StreamArgs st;
  GatedArgs<T> gated;
  DenseOut out;
  const T* w[3];
  const float* bias[3];
  T* y;
  float* y32;
  float* state;
  const int32_t *pos, *seq;
  unsigned long long* key;
  int M, N, ldx, ldw, ldy, lead;
  float limit;
};
// where the rows of a matrix-vector call come from
constexpr int ROWS_GIVEN = 0, ROWS_STREAM = 1, ROWS_GATED = 2;

constexpr int MV_THREADS = 256;
constexpr int MV_WARPS = MV_THREADS / 32;

template <typename T>
__device__ __forceinline__ float dot_chunk(float acc, const uint4& w, const uint4& x) {
  float wf[Elem<T>::VEC], xf[Elem<T>::VEC];
  unpack_chunk(w, wf);
  unpack_chunk(x, xf);
#pragma unroll
  for (int i = 0; i < Elem<T>::VEC; i++) acc = fmaf(wf[i], xf[i], acc);
  return acc;
}

template <typename T, int MT, int EPI, int FROM>
__global__ void __launch_bounds__(MV_THREADS, 2) dense_mv_kernel(const MvArgs<T> a) {
  constexpr int VEC = Elem<T>::VEC;
  constexpr int NW = EPI == JG_DENSE_GLU ? 2 : (EPI == JG_DENSE_MINGRU ? 3 : 1);
  constexpr int RW = NW == 1 ? 2 : 1;    // weight rows per matrix and unit
  constexpr int NACC = NW * RW;
  constexpr int U = MT == 1 ? (NW == 3 ? 5 : 8) : (NW == 3 ? 2 : 4);  // 16-byte loads in flight per lane and weight row
  constexpr int GU = (8 / MT) / (NW == 3 ? 2 : 1);                   // units per cooperative pass
  extern __shared__ __align__(16) unsigned char smem_raw[];
  T* xs = reinterpret_cast<T*>(smem_raw);  // [MT][ldw]
  __shared__ float part[MV_WARPS][GU * NACC * MT];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int N = a.N, KC = a.ldw / VEC;
  pdl_launch();

  const int n_units = (N + RW - 1) / RW;
  const int u0 = (int)((long long)blockIdx.x * n_units / gridDim.x);
  const int u1 = (int)((long long)(blockIdx.x + 1) * n_units / gridDim.x);
  const int nb = (u1 - u0) / MV_WARPS, rem0 = u0 + nb * MV_WARPS;
  const size_t row_bytes = (size_t)a.ldw * sizeof(T);
  auto wrow = [&](int w, int row) { return reinterpret_cast<const unsigned char*>(a.w[w]) + (size_t)row * row_bytes; };

  // weights do not depend on the preceding kernel: the head of this warp's rows travels to L2 while it drains
  if (lane < NACC) {
    const int w = lane / RW, r = lane % RW;
    if (nb > 0) {
      const uint32_t bytes = (uint32_t)min((size_t)4096, row_bytes);
      asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(wrow(w, min((u0 + warp * nb) * RW + r, N - 1))), "r"(bytes) : "memory");
    } else if (rem0 < u1) {
      const size_t off = (size_t)warp * 512;
      if (off + 512 <= row_bytes)
        asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(wrow(w, min(rem0 * RW + r, N - 1)) + off), "r"(512u) : "memory");
    }
  }
  pdl_wait();
  if (EPI == JG_DENSE_STORE && a.out.act == JG_ACT_GELU_SIDE && tid < a.M && u0 < u1)  // this CTA's part of the tokens' rows
    prefetch_l2(dense_side_ptr<T>(a.out, a.out.tokens[tid], u0 * RW));

  for (int m = 0; m < MT; m++) {
    T* xm = xs + (size_t)m * a.ldw;
    if (m >= a.M) {
      for (int c = tid; c < KC; c += MV_THREADS) reinterpret_cast<uint4*>(xm)[c] = make_uint4(0, 0, 0, 0);
    } else if (FROM == ROWS_GATED) {
      float* buf = reinterpret_cast<float*>(smem_raw + (size_t)MT * row_bytes);
      const int n = a.gated.H * a.gated.vd;
      const T* xg = a.x + (size_t)m * a.ldx;
      for (int c = tid; c < a.lead; c += MV_THREADS) xm[c] = xg[c];
      for (int c = a.lead + n + tid; c < a.ldw; c += MV_THREADS) xm[c] = from_f32<T>(0.f);
      if (m > 0) __syncthreads();
      gated_row<MV_THREADS>(a.gated, (size_t)m, buf, [&](int i, const auto& v) {
#pragma unroll
        for (size_t k = 0; k < sizeof(v) / sizeof(float); k++) xm[a.lead + i + k] = from_f32<T>(v[k]);
      });
    } else if (FROM == ROWS_STREAM) {
      float* buf = reinterpret_cast<float*>(smem_raw + (size_t)MT * row_bytes);
      float* red = buf + ((a.st.D + 3) & ~3);
      const size_t src = a.st.rows ? (size_t)a.st.rows[m] : (size_t)m;
      for (int i = a.st.D + tid; i < a.ldw; i += MV_THREADS) xm[i] = from_f32<T>(0.f);
      if (m > 0) __syncthreads();
      stream_row<MV_THREADS>(a.st, src, (blockIdx.x == 0 && a.st.x_out) ? a.st.x_out + src * a.st.D : nullptr, buf, red,
                             [&](int i, const auto& v) {
#pragma unroll
                               for (size_t k = 0; k < sizeof(v) / sizeof(float); k++) xm[i + k] = from_f32<T>(v[k]);
                             });
    } else {
      const T* xg = a.x + (size_t)m * a.ldx;
      for (int c = tid; c < KC; c += MV_THREADS) reinterpret_cast<uint4*>(xm)[c] = ld_128(xg + (size_t)c * VEC);
    }
  }
  __syncthreads();

  unsigned long long best[MT];
#pragma unroll
  for (int m = 0; m < MT; m++) best[m] = 0ull;
  // s: the sums of this output's NW matrices
  auto finish = [&](int row, int m, float s0, float s1, float s2) {
    if (a.bias[0]) s0 += a.bias[0][row];
    const size_t o = (size_t)m * a.ldy + row;
    if (EPI == JG_DENSE_STORE) {
      s0 = dense_act(a.out, row, s0, dense_side<T>(a.out, m, row));
      if (row >= a.out.split) a.out.y2[(size_t)m * a.out.ld2 + row - a.out.split] = s0;
      else if (a.y32) a.y32[o] = s0;
      else a.y[o] = from_f32<T>(s0);
    } else if (EPI == JG_DENSE_GLU) {
      if (a.bias[1]) s1 += a.bias[1][row];
      a.y[o] = from_f32<T>(clamped_glu(s0, s1, a.limit));
    } else if (EPI == JG_DENSE_MINGRU) {
      if (a.bias[1]) s1 += a.bias[1][row];
      float* st = a.state + (size_t)a.seq[m] * N + row;
      const float z = sigmoid_f32(s0), prev = a.pos[m] > 0 ? *st : 0.f;
      const float s = fmaf(z, mingru_candidate(s1), (1.0f - z) * prev);
      *st = s;
      a.y[o] = from_f32<T>(s * silu_f32(s2));
    } else {
      a.y32[o] = s0;
      const unsigned long long k = argmax_key_f32(s0, (uint32_t)row);
#pragma unroll
      for (int q = 0; q < MT; q++)
        if (q == m && k > best[q]) best[q] = k;
    }
  };

  for (int unit = u0 + warp * nb; unit < u0 + (warp + 1) * nb; unit++) {
    float acc[NACC][MT];
    const unsigned char* wp[NACC];
#pragma unroll
    for (int j = 0; j < NACC; j++) {
#pragma unroll
      for (int m = 0; m < MT; m++) acc[j][m] = 0.f;
      wp[j] = wrow(j / RW, min(unit * RW + (j % RW), N - 1));  // clamp: a duplicate row is computed, never stored
    }
    for (int c0 = lane; c0 < KC; c0 += 32 * U) {
      uint4 wv[NACC][U];
#pragma unroll
      for (int u = 0; u < U; u++)
#pragma unroll
        for (int j = 0; j < NACC; j++) wv[j][u] = (c0 + 32 * u < KC) ? ld_stream_128(wp[j] + (size_t)(c0 + 32 * u) * 16) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int u = 0; u < U; u++)
        if (c0 + 32 * u < KC) {
#pragma unroll
          for (int m = 0; m < MT; m++) {
            const uint4 xv = reinterpret_cast<const uint4*>(xs + (size_t)m * a.ldw)[c0 + 32 * u];
#pragma unroll
            for (int j = 0; j < NACC; j++) acc[j][m] = dot_chunk<T>(acc[j][m], wv[j][u], xv);
          }
        }
    }
#pragma unroll
    for (int j = 0; j < NACC; j++)
#pragma unroll
      for (int m = 0; m < MT; m++) acc[j][m] = warp_sum(acc[j][m]);
#pragma unroll
    for (int r = 0; r < RW; r++)
#pragma unroll
      for (int m = 0; m < MT; m++)
        if (lane == r * MT + m && unit * RW + r < N && m < a.M)
          finish(unit * RW + r, m, acc[r][m], NW > 1 ? acc[(NW > 1 ? RW : 0) + r][m] : 0.f, NW > 2 ? acc[(NW > 2 ? 2 * RW : 0) + r][m] : 0.f);
  }

  // remainder (< 8 units of the CTA): all warps on the same units, K split between them in 512-byte pieces
  for (int g0 = rem0; g0 < u1; g0 += GU) {
    const int gu = min(GU, u1 - g0);
    float acc[GU * NACC][MT];
#pragma unroll
    for (int j = 0; j < GU * NACC; j++)
#pragma unroll
      for (int m = 0; m < MT; m++) acc[j][m] = 0.f;
    for (int c = warp * 32 + lane; c < KC; c += MV_THREADS) {
      uint4 wv[GU * NACC];
#pragma unroll
      for (int j = 0; j < GU * NACC; j++) {
        const int unit = g0 + j / NACC, jj = j % NACC;
        wv[j] = (j / NACC < gu) ? ld_stream_128(wrow(jj / RW, min(unit * RW + (jj % RW), N - 1)) + (size_t)c * 16) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int m = 0; m < MT; m++) {
        const uint4 xv = reinterpret_cast<const uint4*>(xs + (size_t)m * a.ldw)[c];
#pragma unroll
        for (int j = 0; j < GU * NACC; j++) acc[j][m] = dot_chunk<T>(acc[j][m], wv[j], xv);
      }
    }
#pragma unroll
    for (int j = 0; j < GU * NACC; j++)
#pragma unroll
      for (int m = 0; m < MT; m++) {
        const float v = warp_sum(acc[j][m]);
        if (lane == 0) part[warp][j * MT + m] = v;
      }
    __syncthreads();
    if (tid < gu * RW * MT) {
      const int ul = tid / (RW * MT), r = (tid / MT) % RW, m = tid % MT, row = (g0 + ul) * RW + r;
      if (row < N && m < a.M) {
        float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
        for (int q = 0; q < NW; q++)
#pragma unroll
          for (int w = 0; w < MV_WARPS; w++) s[q] += part[w][(ul * NACC + q * RW + r) * MT + m];
        finish(row, m, s[0], s[1], s[2]);
      }
    }
    __syncthreads();
  }

  if (EPI == JG_DENSE_LOGITS) {
#pragma unroll
    for (int m = 0; m < MT; m++) {
      unsigned long long b = best[m];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const unsigned long long other = __shfl_xor_sync(0xffffffffu, b, o);
        b = other > b ? other : b;
      }
      if (lane == 0 && m < a.M && b != 0ull) atomicMax(a.key + m, b);
    }
  }
}

template <typename T>
static GatedArgs<T> gated_args(const jg_gated_desc& d) {
  GatedArgs<T> g = {};
  g.o = (const float*)d.o; g.den = (const float*)d.den; g.w = (const float*)d.norm_w; g.gate = (const T*)d.gate;
  g.H = d.heads; g.vd = d.vdim; g.groups = d.groups; g.ldp = d.ldp; g.eps = d.eps; g.scale = d.scale;
  g.vec = d.vdim % 4 == 0 && d.heads * d.vdim / d.groups % 4 == 0 && d.ldp % 4 == 0 && d.gate % (4 * sizeof(T)) == 0 && d.o % 16 == 0 && d.norm_w % 16 == 0;
  return g;
}
static size_t gated_smem_floats(const jg_gated_desc& d, int warps) { return 2 * (size_t)((d.heads * d.vdim + 3) & ~3) + stream_units(d.groups, warps); }

template <typename T, int MT, int EPI, int FROM>
static int launch_mv(jg_dev* dev, const DenseCall& c) {
  auto kern = dense_mv_kernel<T, MT, EPI, FROM>;
  constexpr int RW = (EPI == JG_DENSE_GLU || EPI == JG_DENSE_MINGRU) ? 1 : 2;
  MvArgs<T> a = {};
  a.x = (const T*)c.x; a.st = c.st;
  for (int i = 0; i < 3; i++) { a.w[i] = (const T*)c.w[i]; a.bias[i] = c.bias[i]; }
  if (c.out_f32) a.y32 = (float*)c.y;
  else a.y = (T*)c.y;
  a.state = c.state; a.pos = c.pos; a.seq = c.seq; a.key = c.key;
  a.M = c.M; a.N = c.N; a.ldx = c.ldx; a.ldw = c.ldw; a.ldy = c.ldy; a.limit = c.limit; a.out = c.out; a.lead = c.lead;
  if (FROM == ROWS_GATED) a.gated = gated_args<T>(*c.gated);
  const size_t smem = (size_t)MT * c.ldw * sizeof(T) + (FROM == ROWS_STREAM  ? stream_smem_floats(c.st.D, c.st.groups, MV_WARPS) * sizeof(float)
                                                        : FROM == ROWS_GATED ? gated_smem_floats(*c.gated, MV_WARPS) * sizeof(float) : 0);
  const size_t limit = (size_t)dev->prop.sharedMemPerBlockOptin - 8192;
  if (smem > limit) {
    jg_set_error("dense: %d rows of K=%d need %zu B of shared memory (limit %zu)", MT, c.K, smem, limit);
    return JG_ENOTSUP;
  }
  static bool set[8] = {};
  static size_t occ_smem[8] = {};
  static int occ_for[8] = {};
  const int slot = dev->ordinal & 7;
  if (!set[slot]) {
    JG_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit));
    set[slot] = true;
  }
  if (occ_for[slot] == 0 || occ_smem[slot] != smem) {
    int occ = 0;
    JG_CUDA(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, kern, MV_THREADS, smem));
    occ_for[slot] = occ < 1 ? 1 : (occ > 4 ? 4 : occ);
    occ_smem[slot] = smem;
  }
  const int n_units = (c.N + RW - 1) / RW;
  long long blocks = (long long)dev->sm_count * occ_for[slot];
  if (blocks > n_units) blocks = n_units;
  return jg_launch(dev, "dense_mv", kern, dim3((unsigned)blocks), dim3(MV_THREADS), smem, a);
}

// ------------------------------------------------------------------------------------------------ fp32, many rows
// 64 x 64 output tile, 4 x 4 per thread, plain fp32 FMAs; blocks of 16 k are summed by themselves and then added up.
__global__ void __launch_bounds__(256) dense_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ bias,
                                                        float* __restrict__ y, int M, int N, int K, int ldx, int ldw, int ldy, const DenseOut out) {
  __shared__ float xs[16][65], ws[16][65];
  pdl_launch();
  pdl_wait();
  const int tid = threadIdx.x, tm = tid / 16, tn = tid % 16, m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = tid; i < 64 * 16; i += 256) {
      const int r = i / 16, k = i % 16;
      xs[k][r] = (m0 + r < M && k0 + k < K) ? x[(size_t)(m0 + r) * ldx + k0 + k] : 0.f;
      ws[k][r] = (n0 + r < N && k0 + k < K) ? w[(size_t)(n0 + r) * ldw + k0 + k] : 0.f;
    }
    __syncthreads();
    float part[4][4] = {};
#pragma unroll
    for (int k = 0; k < 16; k++)
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) part[i][j] = fmaf(xs[k][tm + 16 * i], ws[k][tn + 16 * j], part[i][j]);
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) acc[i][j] += part[i][j];
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int m = m0 + tm + 16 * i, n = n0 + tn + 16 * j;
      if (m >= M || n >= N) continue;
      const float v = dense_act(out, n, acc[i][j] + (bias ? bias[n] : 0.f), dense_side<float>(out, m, n));
      if (n >= out.split) out.y2[(size_t)m * out.ld2 + n - out.split] = v;
      else y[(size_t)m * ldy + n] = v;
    }
}

// y <- clamped_glu(y, u) after two separate projections (fp32 operands)
__global__ void glu_f32_kernel(float* __restrict__ y, const float* __restrict__ u, int M, int N, int ld, int ldu, float limit) {
  pdl_launch();
  pdl_wait();
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < (long long)M * N; i += (long long)gridDim.x * blockDim.x) {
    const int m = (int)(i / N), n = (int)(i % N);
    y[(size_t)m * ld + n] = clamped_glu(y[(size_t)m * ld + n], u[(size_t)m * ldu + n], limit);
  }
}

// (value, lowest index) keys of fp32 rows; one CTA per row
__global__ void __launch_bounds__(256) key_f32_kernel(unsigned long long* __restrict__ key, const float* __restrict__ x, int n, int ld) {
  __shared__ unsigned long long red[8];
  pdl_launch();
  pdl_wait();
  const float* xr = x + (size_t)blockIdx.x * ld;
  unsigned long long b = 0ull;
  for (int i = threadIdx.x; i < n; i += 256) {
    const unsigned long long k = argmax_key_f32(xr[i], (uint32_t)i);
    b = k > b ? k : b;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const unsigned long long other = __shfl_xor_sync(0xffffffffu, b, o);
    b = other > b ? other : b;
  }
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = b;
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int i = 1; i < 8; i++) b = red[i] > b ? red[i] : b;
    key[blockIdx.x] = b;
  }
}

// Rows through the stream step on their own (more rows than the matrix-vector kernel takes).
template <typename T>
__global__ void __launch_bounds__(256) stream_step_kernel(const StreamArgs a, T* __restrict__ h, int ldh) {
  extern __shared__ __align__(16) float sbuf[];
  pdl_launch();
  pdl_wait();
  const size_t r = blockIdx.x, src = a.rows ? (size_t)a.rows[r] : r;
  T* hr = h + r * ldh;
  if (a.w_norm || a.plain)
    for (int i = a.D + threadIdx.x; i < ldh; i += 256) hr[i] = from_f32<T>(0.f);
  stream_row<256>(a, src, a.x_out ? a.x_out + src * a.D : nullptr, sbuf, sbuf + ((a.D + 3) & ~3), [&](int i, const auto& v) {
    constexpr int V = sizeof(v) / sizeof(float);
    if constexpr (V == 4 && sizeof(T) == 2) {
      if (ldh % 4 == 0) {
        __nv_bfloat162 p0 = __floats2bfloat162_rn(v[0], v[1]), p1 = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(hr + i) = make_uint2(*reinterpret_cast<uint32_t*>(&p0), *reinterpret_cast<uint32_t*>(&p1));
        return;
      }
    }
#pragma unroll
    for (int k = 0; k < V; k++) hr[i + k] = from_f32<T>(v[k]);
  });
}

template <typename T>
static int launch_stream(jg_dev* dev, const StreamArgs& st, T* h, int ldh, int R) {
  const size_t smem = stream_smem_floats(st.D, st.groups, 8) * sizeof(float);
  const size_t limit = (size_t)dev->prop.sharedMemPerBlockOptin - 1024;
  if (smem > limit) {
    jg_set_error("norm: rows of %d values need %zu B of shared memory (limit %zu)", st.D, smem, limit);
    return JG_ENOTSUP;
  }
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(stream_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit));
    set[dev->ordinal & 7] = true;
  }
  return jg_launch(dev, "stream_step", stream_step_kernel<T>, dim3((unsigned)R), dim3(256), smem, st, h, ldh);
}

template <typename T>
__global__ void __launch_bounds__(256) stream_embed_kernel(float* __restrict__ out, const int32_t* __restrict__ tokens, const T* __restrict__ table, int dim, int ld, int vocab,
                                                           float scale) {
  pdl_launch();
  pdl_wait();
  const int tok = tokens[blockIdx.x];
  const T* row = table + (size_t)(tok >= 0 && tok < vocab ? tok : 0) * ld;
  const bool in = tok >= 0 && tok < vocab;  // an id outside the table reads as zeros
  float* o = out + (size_t)blockIdx.x * dim;
#pragma unroll 4
  for (int c = threadIdx.x; c < dim; c += 256) o[c] = in ? to_f32(row[c]) * scale : 0.f;
}

// ------------------------------------------------------------------------------------------------ dispatch
template <typename T, int EPI, int FROM>
static int mv_rows(jg_dev* dev, const DenseCall& c) {
  return c.M == 1 ? launch_mv<T, 1, EPI, FROM>(dev, c) : launch_mv<T, 2, EPI, FROM>(dev, c);
}
template <typename T>
static int mv_dispatch(jg_dev* dev, const DenseCall& c) {
  const bool norm = c.x == nullptr;
  switch (c.epilogue) {
    case JG_DENSE_STORE:
      if (c.gated) return mv_rows<T, JG_DENSE_STORE, ROWS_GATED>(dev, c);
      return norm ? mv_rows<T, JG_DENSE_STORE, ROWS_STREAM>(dev, c) : mv_rows<T, JG_DENSE_STORE, ROWS_GIVEN>(dev, c);
    case JG_DENSE_GLU: return norm ? mv_rows<T, JG_DENSE_GLU, ROWS_STREAM>(dev, c) : mv_rows<T, JG_DENSE_GLU, ROWS_GIVEN>(dev, c);
    case JG_DENSE_LOGITS: return norm ? mv_rows<T, JG_DENSE_LOGITS, ROWS_STREAM>(dev, c) : mv_rows<T, JG_DENSE_LOGITS, ROWS_GIVEN>(dev, c);
    case JG_DENSE_MINGRU: if (norm) return mv_rows<T, JG_DENSE_MINGRU, ROWS_STREAM>(dev, c);
  }
  jg_set_error("dense: epilogue %d has no kernel for these operands", c.epilogue);
  return JG_ENOTSUP;
}

static int f32_gemm(jg_dev* dev, const DenseCall& c, const void* w, const float* bias, float* y, int ldy) {
  const dim3 grid((unsigned)((c.N + 63) / 64), (unsigned)((c.M + 63) / 64));
  return jg_launch(dev, "dense_f32", dense_f32_kernel, grid, dim3(256), 0, (const float*)c.x, (const float*)w, bias, y, c.M, c.N, c.K, c.ldx, c.ldw, ldy, c.out);
}

int jg_dense_call(jg_dev* dev, const DenseCall& c) {
  if (c.M <= 2) return c.dtype == JG_F32 ? mv_dispatch<float>(dev, c) : mv_dispatch<bf16>(dev, c);
  JG_REQUIRE(c.gated == nullptr, "dense: %d rows: run jg_gated_norm first and pass its rows", c.M);
  JG_REQUIRE(c.x != nullptr, "dense: %d rows: run the stream step first (jg_stream_norm) and pass its rows", c.M);
  JG_REQUIRE(c.epilogue != JG_DENSE_MINGRU, "dense: the recurrent epilogue takes 1-2 rows (M=%d)", c.M);
  int rc;
  if (c.dtype == JG_BF16) {
    rc = jg_dense_tc(dev, c);
  } else if (c.epilogue == JG_DENSE_GLU) {
    // the linear half goes behind the gate half: the caller's rows are 2 x ldy apart in the fp32 build of the buffer
    rc = f32_gemm(dev, c, c.w[0], c.bias[0], (float*)c.y, c.ldy);
    if (rc) return rc;
    float* u = (float*)c.y + (size_t)c.M * c.ldy;
    rc = f32_gemm(dev, c, c.w[1], c.bias[1], u, c.ldy);
    if (rc) return rc;
    rc = jg_launch(dev, "glu_f32", glu_f32_kernel, dim3((unsigned)(dev->sm_count * 4)), dim3(256), 0, (float*)c.y, (const float*)u, c.M, c.N, c.ldy, c.ldy, c.limit);
  } else {
    rc = f32_gemm(dev, c, c.w[0], c.bias[0], (float*)c.y, c.ldy);
  }
  if (rc || c.epilogue != JG_DENSE_LOGITS) return rc;
  return jg_launch(dev, "key_f32", key_f32_kernel, dim3((unsigned)c.M), dim3(256), 0, c.key, (const float*)c.y, c.N, c.ldy);
}

static int check_batch(const char* name, const jg_batch* b) {
  JG_REQUIRE(b != nullptr && b->B > 0 && b->Sc > 0, "%s: empty batch", name);
  return JG_OK;
}
static int fill_stream(const char* name, const jg_stream_desc& s, StreamArgs* a) {
  JG_REQUIRE(s.width > 0 && s.groups > 0 && s.width % s.groups == 0, "%s: %d values do not divide into %d groups", name, s.width, s.groups);
  JG_REQUIRE(jg_aligned(s.x, 16) && (s.y == 0) == (s.w_add == 0), "%s: bad stream pointers", name);
  a->plain = s.plain;
  for (uint64_t p : {s.y, s.w_add, s.x_out, s.w_norm, s.rows}) JG_REQUIRE(p % (p == s.rows ? 4 : 16) == 0, "%s: misaligned pointer", name);
  a->x = (const float*)s.x; a->y = (const float*)s.y; a->w_add = (const float*)s.w_add; a->x_out = (float*)s.x_out;
  a->w_norm = (const float*)s.w_norm; a->rows = (const int32_t*)s.rows; a->D = s.width; a->groups = s.groups; a->eps = s.eps;
  return JG_OK;
}

JG_API int jg_stream_embed(jg_dev* dev, const jg_batch* b, uint64_t out, uint64_t tokens, uint64_t table, int32_t dtype, int32_t dim, int32_t ld, int32_t vocab, float scale) {
  JG_ENTER(dev);
  int rc = check_batch("stream_embed", b);
  if (rc) return rc;
  JG_REQUIRE(dim > 0 && ld >= dim && vocab > 0 && (dtype == JG_F32 || dtype == JG_BF16), "stream_embed: bad shape");
  JG_REQUIRE(jg_aligned(out, 4) && jg_aligned(tokens, 4) && table != 0, "stream_embed: null or misaligned pointer");
  const dim3 grid((unsigned)(b->B * b->Sc));
  if (dtype == JG_F32)
    return jg_launch(dev, "stream_embed", stream_embed_kernel<float>, grid, dim3(256), 0, (float*)out, (const int32_t*)tokens, (const float*)table, dim, ld, vocab, scale);
  return jg_launch(dev, "stream_embed", stream_embed_kernel<bf16>, grid, dim3(256), 0, (float*)out, (const int32_t*)tokens, (const bf16*)table, dim, ld, vocab, scale);
}

JG_API int jg_stream_norm(jg_dev* dev, const jg_batch* b, const jg_stream_desc* s, uint64_t h, int32_t ldh, int32_t dtype) {
  JG_ENTER(dev);
  int rc = check_batch("stream_norm", b);
  if (rc) return rc;
  JG_REQUIRE(s != nullptr && (dtype == JG_F32 || dtype == JG_BF16), "stream_norm: bad arguments");
  StreamArgs a = {};
  rc = fill_stream("stream_norm", *s, &a);
  if (rc) return rc;
  JG_REQUIRE((s->w_norm == 0 && !s->plain) || (jg_aligned(h, 16) && ldh >= s->width), "stream_norm: bad output");
  const int R = b->B * b->Sc;
  return dtype == JG_F32 ? launch_stream<float>(dev, a, (float*)h, ldh, R) : launch_stream<bf16>(dev, a, (bf16*)h, ldh, R);
}

static int check_gated(const char* name, const jg_gated_desc& d) {
  JG_REQUIRE(d.dtype == JG_F32 || d.dtype == JG_BF16, "%s: unknown element type %d", name, d.dtype);
  JG_REQUIRE(d.heads > 0 && d.vdim > 0 && d.groups > 0 && d.heads * d.vdim % d.groups == 0 && d.ldp >= d.heads * d.vdim, "%s: bad gated row", name);
  JG_REQUIRE(jg_aligned(d.o, 4) && d.den % 4 == 0 && d.gate && jg_aligned(d.norm_w, 4), "%s: null or misaligned pointer", name);
  return JG_OK;
}

// Gated rows on their own (more rows than the matrix-vector kernel takes).
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedArgs<T> a, T* __restrict__ out, int ldo) {
  extern __shared__ __align__(16) float sbuf[];
  pdl_launch();
  pdl_wait();
  const size_t r = blockIdx.x;
  gated_row<256>(a, r, sbuf, [&](int i, const auto& v) {
    constexpr int V = sizeof(v) / sizeof(float);
    if constexpr (V == 4 && sizeof(T) == 2) {
      if (ldo % 4 == 0 && (uintptr_t)out % 8 == 0) {
        const __nv_bfloat162 p0 = __floats2bfloat162_rn(v[0], v[1]), p1 = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(out + r * ldo + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&p0), *reinterpret_cast<const uint32_t*>(&p1));
        return;
      }
    }
#pragma unroll
    for (int k = 0; k < V; k++) out[r * ldo + i + k] = from_f32<T>(v[k]);
  });
}
template <typename T>
static int launch_gated(jg_dev* dev, const jg_gated_desc& d, T* out, int ldo, int R) {
  const size_t smem = gated_smem_floats(d, 8) * sizeof(float), limit = (size_t)dev->prop.sharedMemPerBlockOptin - 1024;
  if (smem > limit) {
    jg_set_error("gated_norm: rows of %d values need %zu B of shared memory (limit %zu)", d.heads * d.vdim, smem, limit);
    return JG_ENOTSUP;
  }
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(gated_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)limit));
    set[dev->ordinal & 7] = true;
  }
  return jg_launch(dev, "gated_norm", gated_norm_kernel<T>, dim3((unsigned)R), dim3(256), smem, gated_args<T>(d), out, ldo);
}
JG_API int jg_gated_norm(jg_dev* dev, const jg_batch* b, const jg_gated_desc* d, uint64_t out, int32_t ldo) {
  JG_ENTER(dev);
  int rc = check_batch("gated_norm", b);
  if (rc) return rc;
  JG_REQUIRE(d != nullptr, "gated_norm: null descriptor");
  rc = check_gated("gated_norm", *d);
  if (rc) return rc;
  JG_REQUIRE(out != 0 && out % (d->dtype == JG_F32 ? 4 : 2) == 0 && ldo >= d->heads * d->vdim, "gated_norm: bad output");
  const int R = b->B * b->Sc;
  return d->dtype == JG_F32 ? launch_gated<float>(dev, *d, (float*)out, ldo, R) : launch_gated<bf16>(dev, *d, (bf16*)out, ldo, R);
}

JG_API int jg_dense(jg_dev* dev, const jg_batch* b, const jg_dense_desc* d) {
  JG_ENTER(dev);
  int rc = check_batch("dense", b);
  if (rc) return rc;
  JG_REQUIRE(d != nullptr && (d->dtype == JG_F32 || d->dtype == JG_BF16), "dense: bad arguments");
  const int vec = d->dtype == JG_F32 ? 4 : 8;
  JG_REQUIRE(d->N > 0 && d->K > 0 && d->ldw >= d->K && d->ldw % vec == 0 && d->ldy >= d->N, "dense: bad shape N=%d K=%d ldw=%d ldy=%d", d->N, d->K, d->ldw, d->ldy);
  DenseCall c = {};
  c.dtype = d->dtype; c.epilogue = d->epilogue; c.M = b->B * b->Sc; c.N = d->N; c.K = d->K;
  c.x = (const void*)d->x; c.ldx = d->ldx; c.ldw = d->ldw; c.ldy = d->ldy; c.out_f32 = d->out_f32; c.limit = d->limit;
  const uint64_t w[3] = {d->w0, d->w1, d->w2}, bias[3] = {d->b0, d->b1, d->b2};
  const int nw = d->epilogue == JG_DENSE_GLU ? 2 : (d->epilogue == JG_DENSE_MINGRU ? 3 : 1);
  for (int i = 0; i < 3; i++) {
    JG_REQUIRE(i >= nw || jg_aligned(w[i], 16), "dense: null or misaligned weight");
    JG_REQUIRE(bias[i] % 4 == 0, "dense: misaligned bias");
    c.w[i] = (const void*)w[i]; c.bias[i] = (const float*)bias[i];
  }
  JG_REQUIRE(d->y != 0 && d->y % 4 == 0, "dense: null or misaligned output");
  c.y = (void*)d->y;
  c.out.act = d->act; c.out.lo = d->act_lo; c.out.hi = d->act_hi > 0 ? d->act_hi : d->N; c.out.split = d->split > 0 ? d->split : d->N;
  c.out.ld2 = d->ld2; c.out.y2 = (float*)d->y2; c.out.side = (const void*)d->side; c.out.tokens = (const int32_t*)d->tokens;
  c.out.ld_side = d->ld_side; c.out.col_side = d->col_side; c.out.vocab = d->vocab;
  if (d->epilogue == JG_DENSE_STORE) {
    JG_REQUIRE(d->act >= JG_ACT_NONE && d->act <= JG_ACT_GELU_SIDE && d->act_lo >= 0 && d->split >= 0, "dense: bad activation or split");
    JG_REQUIRE(c.out.split >= d->N || (jg_aligned(d->y2, 4) && d->ld2 >= d->N - c.out.split), "dense: bad fp32 columns");
    JG_REQUIRE(d->act != JG_ACT_GELU_SIDE || (d->side && jg_aligned(d->tokens, 4) && d->col_side >= 0 && d->vocab > 0 && d->ld_side >= d->col_side + d->N), "dense: bad side table");
  }
  if (d->gated.o) {
    const jg_gated_desc& g = d->gated;
    rc = check_gated("dense", g);
    if (rc) return rc;
    JG_REQUIRE(d->epilogue == JG_DENSE_STORE && g.dtype == d->dtype && d->lead >= 0 && d->lead + g.heads * g.vdim == d->K, "dense: the gated prologue needs K = lead + heads * vdim");
    JG_REQUIRE(d->lead == 0 || (jg_aligned(d->x, 16) && d->ldx >= d->lead), "dense: bad leading columns");
    c.gated = &g; c.lead = d->lead;
  } else if (d->x) {
    JG_REQUIRE(jg_aligned(d->x, 16) && d->ldx >= d->ldw && d->ldx % vec == 0, "dense: misaligned rows or row stride (ldx=%d, ldw=%d)", d->ldx, d->ldw);
  } else {
    rc = fill_stream("dense", d->stream, &c.st);
    if (rc) return rc;
    JG_REQUIRE(c.st.D == d->K && (c.st.w_norm != nullptr || c.st.plain) && c.st.x_out != c.st.x, "dense: the stream prologue needs K-wide rows and a second stream buffer");
  }
  if (d->epilogue == JG_DENSE_LOGITS) {
    JG_REQUIRE(jg_aligned(d->key, 8) && d->out_f32, "dense: logits are fp32 and need their keys");
    c.key = (unsigned long long*)d->key;
  }
  if (d->epilogue == JG_DENSE_MINGRU) {
    JG_REQUIRE(jg_aligned(d->state, 4) && jg_aligned(b->pos, 4) && jg_aligned(b->seq, 4) && b->Sc == 1, "dense: the recurrent epilogue needs state, positions and slots, one token per row");
    c.state = (float*)d->state; c.pos = (const int32_t*)b->pos; c.seq = (const int32_t*)b->seq;
  }
  return jg_dense_call(dev, c);
}
