// Recurrent mixers of the layer-list models: the minGRU scan and the gated delta rule, for one token or for a portion of a
// prompt, from and to per-slot state in fp32.  A sequence that starts at position 0 starts from zero whatever its slot
// holds, so a slot needs no clearing between requests.
#include <cooperative_groups.h>

#include "stream.cuh"

namespace cg = cooperative_groups;

// ------------------------------------------------------------------------------------------------ minGRU
// S_t = (1 - z_t) S_{t-1} + z_t c_t is, per channel, an affine map of the state; maps compose, so a portion is scanned in
// blocks of MG_WARPS x MG_TOK tokens: warp w composes its MG_TOK consecutive tokens, the warps' maps meet in shared
// memory, and each warp replays its tokens from the state its predecessors leave.  One CTA = 32 channels of a sequence.
constexpr int MG_WARPS = 32, MG_TOK = 4, MG_THREADS = 32 * MG_WARPS;

template <typename T>
__global__ void __launch_bounds__(MG_THREADS, 1) mingru_scan_kernel(const T* __restrict__ proj, float* __restrict__ state, T* __restrict__ out, const int32_t* __restrict__ pos,
                                                                    const int32_t* __restrict__ seq, int B, int Sc, int width, int ldp, int ldo) {
  __shared__ float s_a[MG_WARPS][32], s_b[MG_WARPS][32], s_carry[2][32];
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, b = blockIdx.y, ch = blockIdx.x * 32 + lane;
  const bool ok = ch < width;
  float* st = state + (size_t)seq[b] * width + ch;
  if (warp == 0) s_carry[0][lane] = (ok && pos[b] > 0) ? *st : 0.f;
  int par = 0;
  T nz[MG_TOK], nc[MG_TOK], ng[MG_TOK];  // the next block's inputs travel while this one is worked on
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < MG_TOK; i++) {
      const int t = t0 + warp * MG_TOK + i;
      if (!ok || t >= Sc) continue;
      const T* p = proj + ((size_t)t * B + b) * ldp + ch;
      nz[i] = p[0]; nc[i] = p[width]; ng[i] = p[2 * width];
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < Sc; t0 += MG_WARPS * MG_TOK) {
    float z[MG_TOK], c[MG_TOK], g[MG_TOK];
    float A = 1.f, Bc = 0.f;
#pragma unroll
    for (int i = 0; i < MG_TOK; i++) {
      const bool in = ok && t0 + warp * MG_TOK + i < Sc;
      z[i] = in ? sigmoid_f32(to_f32(nz[i])) : 0.f;  // past the end: the identity map
      c[i] = in ? z[i] * mingru_candidate(to_f32(nc[i])) : 0.f;
      g[i] = in ? to_f32(ng[i]) : 0.f;
      A *= 1.0f - z[i];
      Bc = fmaf(1.0f - z[i], Bc, c[i]);
    }
    fetch(t0 + MG_WARPS * MG_TOK);
    s_a[warp][lane] = A;
    s_b[warp][lane] = Bc;
    __syncthreads();
    float s = s_carry[par][lane];
    for (int w = 0; w < warp; w++) s = fmaf(s_a[w][lane], s, s_b[w][lane]);
    if (warp == MG_WARPS - 1) s_carry[par ^ 1][lane] = fmaf(A, s, Bc);
#pragma unroll
    for (int i = 0; i < MG_TOK; i++) {
      const int t = t0 + warp * MG_TOK + i;
      s = fmaf(1.0f - z[i], s, c[i]);
      if (ok && t < Sc) out[((size_t)t * B + b) * ldo + ch] = from_f32<T>(s * silu_f32(g[i]));
    }
    par ^= 1;
    __syncthreads();
  }
  if (warp == 0 && ok) *st = s_carry[par][lane];
}

// One token per sequence: one thread per channel.
template <typename T>
__global__ void __launch_bounds__(256) mingru_step_kernel(const T* __restrict__ proj, float* __restrict__ state, T* __restrict__ out, const int32_t* __restrict__ pos,
                                                          const int32_t* __restrict__ seq, int width, int ldp, int ldo) {
  pdl_launch();
  pdl_wait();
  const int ch = blockIdx.x * 256 + threadIdx.x, b = blockIdx.y;
  if (ch >= width) return;
  const T* p = proj + (size_t)b * ldp + ch;
  float* st = state + (size_t)seq[b] * width + ch;
  const float z = sigmoid_f32(to_f32(p[0])), s = fmaf(z, mingru_candidate(to_f32(p[width])), (1.0f - z) * (pos[b] > 0 ? *st : 0.f));
  *st = s;
  out[(size_t)b * ldo + ch] = from_f32<T>(s * silu_f32(to_f32(p[2 * width])));
}

template <typename T>
static int mingru_run(jg_dev* dev, const jg_batch* b, const jg_mingru_desc* d) {
  const int32_t *pos = (const int32_t*)b->pos, *seq = (const int32_t*)b->seq;
  if (b->Sc == 1)
    return jg_launch(dev, "mingru_step", mingru_step_kernel<T>, dim3((unsigned)((d->width + 255) / 256), (unsigned)b->B), dim3(256), 0, (const T*)d->proj, (float*)d->state,
                     (T*)d->out, pos, seq, d->width, d->ldp, d->ldo);
  return jg_launch(dev, "mingru_scan", mingru_scan_kernel<T>, dim3((unsigned)((d->width + 31) / 32), (unsigned)b->B), dim3(MG_THREADS), 0, (const T*)d->proj, (float*)d->state,
                   (T*)d->out, pos, seq, b->B, b->Sc, d->width, d->ldp, d->ldo);
}

static int check_rows(const char* name, const jg_batch* b, int dtype) {
  JG_REQUIRE(b != nullptr && b->B > 0 && b->Sc > 0 && jg_aligned(b->pos, 4) && jg_aligned(b->seq, 4), "%s: bad batch", name);
  JG_REQUIRE(dtype == JG_F32 || dtype == JG_BF16, "%s: unknown element type %d", name, dtype);
  return JG_OK;
}

JG_API int jg_mingru_scan(jg_dev* dev, const jg_batch* b, const jg_mingru_desc* d) {
  JG_ENTER(dev);
  JG_REQUIRE(d != nullptr, "mingru_scan: null descriptor");
  int rc = check_rows("mingru_scan", b, d->dtype);
  if (rc) return rc;
  JG_REQUIRE(d->width > 0 && d->ldp >= 3 * d->width && d->ldo >= d->width && d->proj && d->out && jg_aligned(d->state, 4), "mingru_scan: bad shape or pointer");
  return d->dtype == JG_F32 ? mingru_run<float>(dev, b, d) : mingru_run<bf16>(dev, b, d);
}

// ------------------------------------------------------------------------------------------------ gated delta rule
template <typename T>
struct DeltaArgs {
  const T* proj;
  const float *conv_w, *a_log, *dt_bias, *norm_w;
  float* state;
  T* tail;
  // scratch: unit vectors [R][G][q | k][lds], [R][H][2] (decay, beta), v and then the read-outs [R][H * vd]
  float *qk, *gates, *v, *o;
  T* out;
  const int32_t *pos, *seq;
  int B, Sc, H, G, dim, vd, taps, ldp, ldo, lds;  // lds: dim rounded up to 4
  float eps;
  __device__ __forceinline__ int channels() const { return 2 * G * dim + H * vd; }
  // column of the projection that holds b / a of head h, and the output gate
  __device__ __forceinline__ int col_b() const { return channels(); }
  __device__ __forceinline__ int col_a() const { return channels() + H; }
  __device__ __forceinline__ int col_g() const { return channels() + 2 * H; }
};

// Convolution input of channel c at `back` tokens before token s of sequence b: from this call's rows, from the tail the
// earlier calls left, or zero before the start.
template <typename T>
__device__ __forceinline__ float delta_conv_silu(const DeltaArgs<T>& a, int b, int s, int c, int p0, const T* tail) {
  const float* w = a.conv_w + (size_t)c * a.taps;
  float acc = 0.f;
  for (int j = 0; j < a.taps; j++) {  // j = 0: the oldest tap
    const int back = a.taps - 1 - j, src = s - back;
    float v = 0.f;
    if (src >= 0) v = to_f32(a.proj[((size_t)src * a.B + b) * a.ldp + c]);
    else if (p0 + src >= 0) v = to_f32(tail[(size_t)((p0 + src) % a.taps) * a.channels() + c]);
    acc = fmaf(w[j], v, acc);
  }
  return silu_f32(acc);
}
template <typename T>
__device__ __forceinline__ float2 delta_gates(const DeltaArgs<T>& a, size_t row, int h) {
  const T* p = a.proj + row * a.ldp;
  const float beta = sigmoid_f32(to_f32(p[a.col_b() + h]));
  const float dt = softplus_f32(to_f32(p[a.col_a() + h]) + a.dt_bias[h]);
  return make_float2(expf(-expf(a.a_log[h]) * dt), beta);
}
constexpr float DELTA_UNIT_EPS = 1e-6f;

// Portions, step 1, one CTA per row: convolutions, unit vectors and gates into scratch.
template <typename T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaArgs<T> a) {
  extern __shared__ __align__(16) float buf[];
  pdl_launch();
  pdl_wait();
  const int r = blockIdx.x, b = r % a.B, s = r / a.B, C = a.channels(), p0 = a.pos[b];
  const T* tail = a.tail + (size_t)a.seq[b] * a.taps * C;
  const int nqk = 2 * a.G * a.dim;
  float* dv = a.v + (size_t)r * a.H * a.vd;
#pragma unroll 2
  for (int c = threadIdx.x; c < C; c += 256) {
    const float v = delta_conv_silu(a, b, s, c, p0, tail);
    if (c < nqk) buf[c] = v;
    else dv[c - nqk] = v;
  }
  for (int h = threadIdx.x; h < a.H; h += 256) *reinterpret_cast<float2*>(a.gates + ((size_t)r * a.H + h) * 2) = delta_gates(a, r, h);
  __syncthreads();
  const int lane = threadIdx.x & 31;
  for (int g = threadIdx.x >> 5; g < 2 * a.G; g += 8) {  // q heads, then k heads
    const float* x = buf + g * a.dim;
    float ss = 0.f;
    for (int i = lane; i < a.dim; i += 32) ss = fmaf(x[i], x[i], ss);
    const float rs = 1.0f / sqrtf(warp_sum(ss) + DELTA_UNIT_EPS) * (g < a.G ? 1.0f / sqrtf((float)a.dim) : 1.0f);
    float* dst = a.qk + (((size_t)r * a.G + (g < a.G ? g : g - a.G)) * 2 + (g < a.G ? 0 : 1)) * a.lds;
    for (int i = lane; i < a.lds; i += 32) dst[i] = i < a.dim ? x[i] * rs : 0.f;
  }
}

// One column of S (state transposed: lds consecutive floats), spread over LPC lanes, E elements each: lane l holds the
// float4s l, l + LPC, l + 2 LPC, ...
template <int LPC, int E>
struct DeltaCol {
  float s[E];
  __device__ __forceinline__ void load(const float* p, int l, int lds, bool live) {
#pragma unroll
    for (int i = 0; i < E / 4; i++) {
      const int off = (l + LPC * i) * 4;
      const float4 v = (live && off < lds) ? *reinterpret_cast<const float4*>(p + off) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[4 * i] = v.x; s[4 * i + 1] = v.y; s[4 * i + 2] = v.z; s[4 * i + 3] = v.w;
    }
  }
  __device__ __forceinline__ void store(float* p, int l, int lds) const {
#pragma unroll
    for (int i = 0; i < E / 4; i++) {
      const int off = (l + LPC * i) * 4;
      if (off < lds) *reinterpret_cast<float4*>(p + off) = make_float4(s[4 * i], s[4 * i + 1], s[4 * i + 2], s[4 * i + 3]);
    }
  }
  // one token; kv, qv: this lane's elements of k and q.  The read-out uses S_new^T q = g (S^T q) + (k.q) u, so that both
  // dot products run on the old state, side by side.
  __device__ __forceinline__ float step(const float4 (&kv)[E / 4], const float4 (&qv)[E / 4], float v, float g, float beta, float kq) {
    float dk[2] = {0.f, 0.f}, dq[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < E / 4; i++) {
      const int c = i & 1;
      dk[c] = fmaf(s[4 * i], kv[i].x, dk[c]); dq[c] = fmaf(s[4 * i], qv[i].x, dq[c]);
      dk[c] = fmaf(s[4 * i + 1], kv[i].y, dk[c]); dq[c] = fmaf(s[4 * i + 1], qv[i].y, dq[c]);
      dk[c] = fmaf(s[4 * i + 2], kv[i].z, dk[c]); dq[c] = fmaf(s[4 * i + 2], qv[i].z, dq[c]);
      dk[c] = fmaf(s[4 * i + 3], kv[i].w, dk[c]); dq[c] = fmaf(s[4 * i + 3], qv[i].w, dq[c]);
    }
    float sk = dk[0] + dk[1], sq = dq[0] + dq[1];
#pragma unroll
    for (int o = LPC / 2; o > 0; o >>= 1) { sk += __shfl_xor_sync(0xffffffffu, sk, o); sq += __shfl_xor_sync(0xffffffffu, sq, o); }
    const float u = beta * (v - g * sk);
#pragma unroll
    for (int i = 0; i < E / 4; i++) {
      s[4 * i] = fmaf(kv[i].x, u, g * s[4 * i]);
      s[4 * i + 1] = fmaf(kv[i].y, u, g * s[4 * i + 1]);
      s[4 * i + 2] = fmaf(kv[i].z, u, g * s[4 * i + 2]);
      s[4 * i + 3] = fmaf(kv[i].w, u, g * s[4 * i + 3]);
    }
    return fmaf(u, kq, g * sq);
  }
};

// Portions, step 2: the recurrence.  Columns of S never meet, so a CTA takes DS_COLS columns of one head of one sequence
// and walks the tokens, DS_STEP at a time.  With D_i the product of the decays up to token i of such a group and w_j the
// update of token j decayed to the present one,
//   S_0^T k_i, S_0^T q_i          for all i at once, on the state before the group
//   u_i = beta_i (v_i - D_i S_0^T k_i - sum_{j<i} (k_j . k_i) w_j),   o_i = D_i S_0^T q_i + sum_{j<=i} (k_j . q_i) w_j
//   S   = D S_0 + sum_j k_j w_j^T
// so that the reductions over the lanes of a column overlap instead of following one another.  Blocks of DS_TOK tokens are
// staged by cp.async, one ahead; the products k_j . k_i and k_j . q_i of a block are worked out by all threads first.
constexpr int DS_LPC = 8, DS_COLS = 16, DS_THREADS = DS_LPC * DS_COLS, DS_TOK = 16, DS_STEP = 4, DS_PAIRS = DS_STEP * DS_STEP;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async4(void* smem, const void* gmem) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async8(void* smem, const void* gmem) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}
// two fp32 FMAs in one instruction
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n\t.reg .b64 ra, rb, rc, rd;\n\tmov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\tmov.b64 rc, {%6, %7};\n\t"
      "fma.rn.f32x2 rd, ra, rb, rc;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) { return fma2(a, b, make_float2(-0.0f, -0.0f)); }

template <int E>
struct DeltaStage {
  static constexpr int ROW = E * DS_LPC + 4;  // padded: the rows a warp compares start in different banks
  float k[DS_TOK][ROW], q[DS_TOK][ROW], v[DS_TOK][DS_COLS], gate[DS_TOK][2];
};

template <typename T, int E>
__global__ void __launch_bounds__(DS_THREADS) delta_scan_kernel(const DeltaArgs<T> a) {
  using Stage = DeltaStage<E>;
  extern __shared__ __align__(16) unsigned char dsm[];
  Stage* stages = reinterpret_cast<Stage*>(dsm);
  __shared__ __align__(16) float pairs[DS_TOK / DS_STEP][2][DS_PAIRS];  // [group][k.k | k.q][i * DS_STEP + j]
  pdl_launch();
  const int tid = threadIdx.x, l = tid % DS_LPC, col = tid / DS_LPC, h = blockIdx.y, b = blockIdx.z;
  const int j0 = blockIdx.x * DS_COLS, j = j0 + col, g = h / (a.H / a.G), C = a.channels();
  for (int i = tid; i < (int)(2 * sizeof(Stage) / 4); i += DS_THREADS) reinterpret_cast<float*>(dsm)[i] = 0.f;  // padding, columns past vd
  __syncthreads();
  pdl_wait();
  const int slot = a.seq[b];
  const bool live = j < a.vd;
  const int c4 = a.lds / 4;
  auto stage_block = [&](int t0, Stage& st) {
    const int nt = min(DS_TOK, a.Sc - t0);
    for (int i = tid; i < DS_TOK * 2 * c4; i += DS_THREADS) {
      const int t = i / (2 * c4), e = i % (2 * c4);
      float* dst = e < c4 ? &st.q[t][e * 4] : &st.k[t][(e - c4) * 4];
      if (t < nt) cp_async16(dst, a.qk + (((size_t)(t0 + t) * a.B + b) * a.G + g) * 2 * a.lds + e * 4);
      else *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int i = tid; i < DS_TOK * DS_COLS; i += DS_THREADS) {
      const int t = i / DS_COLS, c = i % DS_COLS;
      if (t < nt && j0 + c < a.vd) cp_async4(&st.v[t][c], a.v + ((size_t)(t0 + t) * a.B + b) * a.H * a.vd + (size_t)h * a.vd + j0 + c);
    }
    if (tid < DS_TOK) {  // a token past the end keeps the state: decay 1, beta 0
      if (tid < nt) cp_async8(st.gate[tid], a.gates + (((size_t)(t0 + tid) * a.B + b) * a.H + h) * 2);
      else { st.gate[tid][0] = 1.f; st.gate[tid][1] = 0.f; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage_block(0, stages[0]);
  float* stp = a.state + (((size_t)slot * a.H + h) * a.vd + (live ? j : 0)) * a.lds;
  DeltaCol<DS_LPC, E> col_s;
  col_s.load(stp, l, a.lds, live && a.pos[b] > 0);
  float2 S[E / 2];
#pragma unroll
  for (int i = 0; i < E / 2; i++) S[i] = make_float2(col_s.s[2 * i], col_s.s[2 * i + 1]);

  int buf = 0;
  for (int t0 = 0; t0 < a.Sc; t0 += DS_TOK, buf ^= 1) {
    if (t0 + DS_TOK < a.Sc) {
      stage_block(t0 + DS_TOK, stages[buf ^ 1]);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const Stage& st = stages[buf];
    // k_j . k_i and k_j . q_i: DS_TOK / DS_STEP groups x 16 pairs, two threads per pair (which share both products)
    {
      const int pr = tid >> 1, half = tid & 1, grp = pr / DS_PAIRS, i = (pr / DS_STEP) % DS_STEP, jj = pr % DS_STEP;
      float dk = 0.f, dq = 0.f;
      if (jj <= i) {
        const float *kj = st.k[grp * DS_STEP + jj], *ki = st.k[grp * DS_STEP + i], *qi = st.q[grp * DS_STEP + i];
        for (int e = half; e < c4; e += 2) {
          const float4 x = *reinterpret_cast<const float4*>(kj + e * 4), y = *reinterpret_cast<const float4*>(ki + e * 4), z = *reinterpret_cast<const float4*>(qi + e * 4);
          dk = fmaf(x.x, y.x, dk); dk = fmaf(x.y, y.y, dk); dk = fmaf(x.z, y.z, dk); dk = fmaf(x.w, y.w, dk);
          dq = fmaf(x.x, z.x, dq); dq = fmaf(x.y, z.y, dq); dq = fmaf(x.z, z.z, dq); dq = fmaf(x.w, z.w, dq);
        }
      }
      dk += __shfl_xor_sync(0xffffffffu, dk, 1);
      dq += __shfl_xor_sync(0xffffffffu, dq, 1);
      if (half == 0) { pairs[grp][0][i * DS_STEP + jj] = dk; pairs[grp][1][i * DS_STEP + jj] = dq; }
    }
    __syncthreads();
    for (int grp = 0; grp < DS_TOK / DS_STEP; grp++) {
      const int tb = grp * DS_STEP;
      float sk[DS_STEP], sq[DS_STEP];
#pragma unroll
      for (int i = 0; i < DS_STEP; i++) {
        float2 ak = make_float2(0.f, 0.f), aq = make_float2(0.f, 0.f);
#pragma unroll
        for (int e = 0; e < E / 4; e++) {
          const float4 kv = *reinterpret_cast<const float4*>(&st.k[tb + i][(l + DS_LPC * e) * 4]), qv = *reinterpret_cast<const float4*>(&st.q[tb + i][(l + DS_LPC * e) * 4]);
          ak = fma2(S[2 * e], make_float2(kv.x, kv.y), ak); ak = fma2(S[2 * e + 1], make_float2(kv.z, kv.w), ak);
          aq = fma2(S[2 * e], make_float2(qv.x, qv.y), aq); aq = fma2(S[2 * e + 1], make_float2(qv.z, qv.w), aq);
        }
        sk[i] = ak.x + ak.y;
        sq[i] = aq.x + aq.y;
      }
#pragma unroll
      for (int o = DS_LPC / 2; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < DS_STEP; i++) { sk[i] += __shfl_xor_sync(0xffffffffu, sk[i], o); sq[i] += __shfl_xor_sync(0xffffffffu, sq[i], o); }
      float w[DS_STEP], D = 1.f, mine = 0.f;
#pragma unroll
      for (int i = 0; i < DS_STEP; i++) {
        const float2 gt = *reinterpret_cast<const float2*>(st.gate[tb + i]);
        D *= gt.x;
        float pre = D * sk[i], o = D * sq[i];
#pragma unroll
        for (int jj = 0; jj < i; jj++) {
          w[jj] *= gt.x;
          pre = fmaf(pairs[grp][0][i * DS_STEP + jj], w[jj], pre);
          o = fmaf(pairs[grp][1][i * DS_STEP + jj], w[jj], o);
        }
        w[i] = gt.y * (st.v[tb + i][col] - pre);
        o = fmaf(pairs[grp][1][i * DS_STEP + i], w[i], o);
        if (l == i) mine = o;
      }
      const float2 D2 = make_float2(D, D);
#pragma unroll
      for (int e = 0; e < E / 2; e++) S[e] = mul2(S[e], D2);
#pragma unroll
      for (int i = 0; i < DS_STEP; i++) {
        const float2 w2 = make_float2(w[i], w[i]);
#pragma unroll
        for (int e = 0; e < E / 4; e++) {
          const float4 kv = *reinterpret_cast<const float4*>(&st.k[tb + i][(l + DS_LPC * e) * 4]);
          S[2 * e] = fma2(make_float2(kv.x, kv.y), w2, S[2 * e]);
          S[2 * e + 1] = fma2(make_float2(kv.z, kv.w), w2, S[2 * e + 1]);
        }
      }
      const int t = t0 + tb + l;
      if (l < DS_STEP && live && t < a.Sc) a.o[((size_t)t * a.B + b) * a.H * a.vd + (size_t)h * a.vd + j] = mine;
    }
    __syncthreads();  // the other stage is refilled next, and `pairs` is rewritten
  }
#pragma unroll
  for (int i = 0; i < E / 2; i++) { col_s.s[2 * i] = S[i].x; col_s.s[2 * i + 1] = S[i].y; }
  if (live) col_s.store(stp, l, a.lds);
  // the convolution's last inputs: entry position % taps, which no row of this call reads any more
  T* tail = a.tail + (size_t)slot * a.taps * C;
  const int cta = blockIdx.y * gridDim.x + blockIdx.x, ctas = gridDim.x * gridDim.y, keep = min(a.taps - 1, a.Sc);
  for (int i = cta * DS_THREADS + tid; i < keep * C; i += ctas * DS_THREADS) {
    const int s = a.Sc - keep + i / C, c = i % C;
    tail[(size_t)((a.pos[b] + s) % a.taps) * C + c] = a.proj[((size_t)s * a.B + b) * a.ldp + c];
  }
}

// Portions, step 3, one warp per (row, head): norm over the value dimension, norm weight, output gate.
template <typename T>
__global__ void __launch_bounds__(256) delta_out_kernel(const DeltaArgs<T> a, int R) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= (long long)R * a.H) return;
  const int r = (int)(id / a.H), h = (int)(id % a.H);
  const float* o = a.o + (size_t)id * a.vd;
  float ss = 0.f;
  for (int i = lane; i < a.vd; i += 32) ss = fmaf(o[i], o[i], ss);
  const float rs = 1.0f / sqrtf(warp_sum(ss) / (float)a.vd + a.eps);
  const T* gate = a.proj + (size_t)r * a.ldp + a.col_g() + h * a.vd;
  for (int i = lane; i < a.vd; i += 32) a.out[(size_t)r * a.ldo + h * a.vd + i] = from_f32<T>(o[i] * rs * a.norm_w[i] * silu_f32(to_f32(gate[i])));
}

// One token per row, everything in one launch: a cluster of CTAs shares a (row, head), each CTA takes a run of columns of
// S; the sum of squares of the output norm crosses through distributed shared memory.
constexpr int DD_THREADS = 256, DD_COLS = DD_THREADS / DS_LPC, DD_MAX_CLUSTER = 8;

template <typename T, int E>
__global__ void __launch_bounds__(DD_THREADS) delta_step_kernel(const DeltaArgs<T> a) {
  constexpr int DP = E * DS_LPC;
  extern __shared__ __align__(16) float dyn[];  // this CTA's columns: v, then o
  __shared__ __align__(16) float sk[DP], sq[DP];
  __shared__ float red[3][DD_THREADS / 32], s_ss[DD_MAX_CLUSTER];
  cg::cluster_group cluster = cg::this_cluster();
  const int cr = (int)cluster.block_rank(), cs = (int)cluster.num_blocks();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l = tid % DS_LPC, col = tid / DS_LPC, h = blockIdx.y, r = blockIdx.z;
  const int g = h / (a.H / a.G), C = a.channels();
  const int per = (a.vd + cs - 1) / cs, j0 = min(a.vd, cr * per), j1 = min(a.vd, j0 + per);
  asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");  // every CTA of the cluster has started ...
  pdl_launch();
  pdl_wait();
  const int p0 = a.pos[r], slot = a.seq[r];
  T* tail = a.tail + (size_t)slot * a.taps * C;
  T* tail_now = tail + (size_t)(p0 % a.taps) * C;  // no CTA reads this entry: it holds position p0 - taps
  const T* row = a.proj + (size_t)r * a.ldp;
  // the first columns of the state are requested before the convolutions
  DeltaCol<DS_LPC, E> S;
  float* st0 = a.state + ((size_t)slot * a.H + h) * a.vd * a.lds;
  S.load(st0 + (size_t)min(j0 + col, a.vd - 1) * a.lds, l, a.lds, p0 > 0);
  float qv = 0.f, kv = 0.f, pq = 0.f, pk = 0.f, pqk = 0.f;
  for (int i = tid; i < DP; i += DD_THREADS) {
    if (i < a.dim) {
      const int cq = g * a.dim + i, ck = (a.G + g) * a.dim + i;
      qv = delta_conv_silu(a, r, 0, cq, p0, tail);
      kv = delta_conv_silu(a, r, 0, ck, p0, tail);
      pq = fmaf(qv, qv, pq); pk = fmaf(kv, kv, pk); pqk = fmaf(qv, kv, pqk);
      sq[i] = qv; sk[i] = kv;
      if (cr == 0 && h % (a.H / a.G) == 0) { tail_now[cq] = row[cq]; tail_now[ck] = row[ck]; }
    } else {
      sq[i] = 0.f; sk[i] = 0.f;
    }
  }
  for (int j = j0 + tid; j < j1; j += DD_THREADS) {
    const int c = 2 * a.G * a.dim + h * a.vd + j;
    dyn[j - j0] = delta_conv_silu(a, r, 0, c, p0, tail);
    tail_now[c] = row[c];
  }
  pq = warp_sum(pq); pk = warp_sum(pk); pqk = warp_sum(pqk);
  if (lane == 0) { red[0][warp] = pq; red[1][warp] = pk; red[2][warp] = pqk; }
  __syncthreads();
  float tq = 0.f, tk = 0.f, tqk = 0.f;
#pragma unroll
  for (int w = 0; w < DD_THREADS / 32; w++) { tq += red[0][w]; tk += red[1][w]; tqk += red[2][w]; }
  const float rq = 1.0f / sqrtf(tq + DELTA_UNIT_EPS) * (1.0f / sqrtf((float)a.dim)), rk = 1.0f / sqrtf(tk + DELTA_UNIT_EPS);
  const float2 gt = delta_gates(a, r, h);
  float4 k4[E / 4], q4[E / 4];
#pragma unroll
  for (int i = 0; i < E / 4; i++) {
    k4[i] = *reinterpret_cast<const float4*>(&sk[(l + DS_LPC * i) * 4]);
    q4[i] = *reinterpret_cast<const float4*>(&sq[(l + DS_LPC * i) * 4]);
    k4[i].x *= rk; k4[i].y *= rk; k4[i].z *= rk; k4[i].w *= rk;
    q4[i].x *= rq; q4[i].y *= rq; q4[i].z *= rq; q4[i].w *= rq;
  }
  float ss = 0.f;
  for (int jb = j0; jb < j1; jb += DD_COLS) {  // the whole warp takes part in the shuffles
    const int j = jb + col;
    const bool live = j < j1;
    float* st = st0 + (size_t)(live ? j : j0) * a.lds;
    DeltaCol<DS_LPC, E> next;
    if (jb + DD_COLS < j1) next.load(st0 + (size_t)min(j + DD_COLS, j1 - 1) * a.lds, l, a.lds, p0 > 0);
    const float o = S.step(k4, q4, live ? dyn[j - j0] : 0.f, gt.x, gt.y, tqk * rq * rk);
    if (live) {
      S.store(st, l, a.lds);
      if (l == 0) { dyn[j - j0] = o; ss = fmaf(o, o, ss); }
    }
    if (jb + DD_COLS < j1) S = next;
    __syncwarp();
  }
  ss = warp_sum(ss);
  __syncthreads();  // red is reused; dyn holds o
  if (lane == 0) red[0][warp] = ss;
  __syncthreads();
  asm volatile("barrier.cluster.wait.aligned;" ::: "memory");  // ... before its shared memory is written from outside
  if (tid < cs) {
    float t = 0.f;
    for (int w = 0; w < DD_THREADS / 32; w++) t += red[0][w];
    *cluster.map_shared_rank(&s_ss[cr], tid) = t;
  }
  cluster.sync();
  float tot = 0.f;
  for (int c = 0; c < cs; c++) tot += s_ss[c];
  const float rs = 1.0f / sqrtf(tot / (float)a.vd + a.eps);
  const T* gate = row + a.col_g() + h * a.vd;
  for (int j = j0 + tid; j < j1; j += DD_THREADS)
    a.out[(size_t)r * a.ldo + h * a.vd + j] = from_f32<T>(dyn[j - j0] * rs * a.norm_w[j] * silu_f32(to_f32(gate[j])));
}

JG_API int jg_delta_scratch_floats(const jg_delta_desc* d, int32_t rows, uint64_t* out) {
  JG_REQUIRE(d != nullptr && out != nullptr && rows > 0, "delta_scratch_floats: bad arguments");
  const uint64_t R = (uint64_t)rows;
  *out = R * (2ull * d->kv_heads * ((d->dim + 3) & ~3) + 2ull * d->heads * d->vdim + 2ull * d->heads) + 16;
  return JG_OK;
}

template <typename T, int E>
static int delta_launch(jg_dev* dev, const DeltaArgs<T>& a) {
  const int R = a.B * a.Sc;
  if (a.Sc == 1) {
    int cs = 1;
    while (cs < DD_MAX_CLUSTER && cs * DD_COLS < a.vd && R * a.H * cs < 2 * dev->sm_count) cs *= 2;
    const size_t smem = (size_t)((a.vd + cs - 1) / cs) * sizeof(float);
    return jg_launch_cluster(dev, "delta_step", delta_step_kernel<T, E>, dim3((unsigned)cs, (unsigned)a.H, (unsigned)R), dim3(DD_THREADS), smem, cs, a);
  }
  const size_t smem = (size_t)2 * a.G * a.dim * sizeof(float);
  static bool set[8] = {};
  if (!set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(delta_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)dev->prop.sharedMemPerBlockOptin - 1024));
    set[dev->ordinal & 7] = true;
  }
  int rc = jg_launch(dev, "delta_prep", delta_prep_kernel<T>, dim3((unsigned)R), dim3(256), smem, a);
  if (rc) return rc;
  static bool scan_set[8] = {};
  if (!scan_set[dev->ordinal & 7]) {
    JG_CUDA(cudaFuncSetAttribute(delta_scan_kernel<T, E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(2 * sizeof(DeltaStage<E>))));
    scan_set[dev->ordinal & 7] = true;
  }
  rc = jg_launch(dev, "delta_scan", delta_scan_kernel<T, E>, dim3((unsigned)((a.vd + DS_COLS - 1) / DS_COLS), (unsigned)a.H, (unsigned)a.B), dim3(DS_THREADS),
                 2 * sizeof(DeltaStage<E>), a);
  if (rc) return rc;
  return jg_launch(dev, "delta_out", delta_out_kernel<T>, dim3((unsigned)(((long long)R * a.H + 7) / 8)), dim3(256), 0, a, R);
}

template <typename T>
static int delta_run(jg_dev* dev, const jg_batch* b, const jg_delta_desc* d) {
  DeltaArgs<T> a = {};
  a.proj = (const T*)d->proj; a.conv_w = (const float*)d->conv_w; a.a_log = (const float*)d->a_log; a.dt_bias = (const float*)d->dt_bias;
  a.norm_w = (const float*)d->norm_w; a.state = (float*)d->state; a.tail = (T*)d->tail; a.out = (T*)d->out;
  a.pos = (const int32_t*)b->pos; a.seq = (const int32_t*)b->seq;
  a.B = b->B; a.Sc = b->Sc; a.H = d->heads; a.G = d->kv_heads; a.dim = d->dim; a.vd = d->vdim; a.taps = d->taps;
  a.ldp = d->ldp; a.ldo = d->ldo; a.lds = (d->dim + 3) & ~3; a.eps = d->eps;
  const size_t R = (size_t)b->B * b->Sc;
  a.qk = (float*)d->scratch;  // 16-byte rows first, 8-byte pairs next
  a.gates = a.qk + R * d->kv_heads * 2 * a.lds;
  a.v = a.gates + R * d->heads * 2;
  a.o = a.v + R * d->heads * d->vdim;
  if (d->dim <= 32) return delta_launch<T, 4>(dev, a);
  if (d->dim <= 64) return delta_launch<T, 8>(dev, a);
  if (d->dim <= 128) return delta_launch<T, 16>(dev, a);
  if (d->dim <= 256) return delta_launch<T, 32>(dev, a);
  jg_set_error("delta_rule: query / key heads of %d values (largest supported: 256)", d->dim);
  return JG_ENOTSUP;
}

JG_API int jg_delta_rule(jg_dev* dev, const jg_batch* b, const jg_delta_desc* d) {
  JG_ENTER(dev);
  JG_REQUIRE(d != nullptr, "delta_rule: null descriptor");
  int rc = check_rows("delta_rule", b, d->dtype);
  if (rc) return rc;
  JG_REQUIRE(d->heads > 0 && d->kv_heads > 0 && d->heads % d->kv_heads == 0 && d->dim > 0 && d->vdim > 0 && d->taps > 0, "delta_rule: bad shape");
  JG_REQUIRE(d->ldp >= 2 * d->kv_heads * d->dim + 2 * d->heads * d->vdim + 2 * d->heads && d->ldo >= d->heads * d->vdim, "delta_rule: row strides too small");
  JG_REQUIRE(jg_aligned(d->state, 16) && jg_aligned(d->scratch, 16) && d->proj && d->tail && d->out && d->conv_w && d->a_log && d->dt_bias && d->norm_w, "delta_rule: null or misaligned pointer");
  return d->dtype == JG_F32 ? delta_run<float>(dev, b, d) : delta_run<bf16>(dev, b, d);
}
