// Recurrent mixers of the layer-list models: the minGRU scan and the gated delta rule, for one token or for a portion of a
// prompt, from and to per-slot state in fp32.  A sequence that starts at position 0 starts from zero whatever its slot
// holds, so a slot needs no clearing between requests.
#include <cooperative_groups.h>

#include "stream.cuh"

namespace cg = cooperative_groups;

// ------------------------------------------------------------------------------------------------ minGRU
// S_t = (1 - z_t) S_{t-1} + z_t c_t is, per channel, an affine map of the state; maps compose, so a portion is scanned in
// blocks of MG_GROUPS x MG_TOK tokens: a group of lanes composes its MG_TOK consecutive tokens, the groups' maps meet in
// shared memory, the first group runs through them, and each group replays its tokens from the state its predecessors
// leave.  One CTA = 16 channels of a sequence.
constexpr int MG_CH = 16, MG_GROUPS = 32, MG_TOK = 4, MG_THREADS = MG_CH * MG_GROUPS;

template <typename T>
__global__ void __launch_bounds__(MG_THREADS) mingru_scan_kernel(const T* __restrict__ proj, float* __restrict__ state, T* __restrict__ out, const int32_t* __restrict__ pos,
                                                                 const int32_t* __restrict__ seq, int B, int Sc, int width, int ldp, int ldo) {
  __shared__ float s_a[MG_GROUPS][MG_CH], s_b[MG_GROUPS][MG_CH], s_in[MG_GROUPS][MG_CH];
  pdl_wait();  // no early trigger: the next kernel's CTAs would sit on this one's SMs for its whole length
  const int c = threadIdx.x % MG_CH, grp = threadIdx.x / MG_CH, b = blockIdx.y, ch = blockIdx.x * MG_CH + c;
  const bool ok = ch < width;
  float* st = state + (size_t)seq[b] * width + ch;
  float carry = (grp == 0 && ok && pos[b] > 0) ? *st : 0.f;  // first group: the state ahead of the block
  T nz[MG_TOK], nc[MG_TOK], ng[MG_TOK];  // the next block's inputs travel while this one is worked on
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < MG_TOK; i++) {
      const int t = t0 + grp * MG_TOK + i;
      if (!ok || t >= Sc) continue;
      const T* p = proj + ((size_t)t * B + b) * ldp + ch;
      nz[i] = p[0]; nc[i] = p[width]; ng[i] = p[2 * width];
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < Sc; t0 += MG_GROUPS * MG_TOK) {
    float z[MG_TOK], u[MG_TOK], g[MG_TOK];
    float A = 1.f, Bc = 0.f;
#pragma unroll
    for (int i = 0; i < MG_TOK; i++) {
      const bool in = ok && t0 + grp * MG_TOK + i < Sc;
      z[i] = in ? sigmoid_f32(to_f32(nz[i])) : 0.f;  // past the end: the identity map
      u[i] = in ? z[i] * mingru_candidate(to_f32(nc[i])) : 0.f;
      g[i] = in ? to_f32(ng[i]) : 0.f;
      A *= 1.0f - z[i];
      Bc = fmaf(1.0f - z[i], Bc, u[i]);
    }
    fetch(t0 + MG_GROUPS * MG_TOK);
    s_a[grp][c] = A;
    s_b[grp][c] = Bc;
    __syncthreads();
    if (grp == 0) {
#pragma unroll 8
      for (int w = 0; w < MG_GROUPS; w++) {
        s_in[w][c] = carry;
        carry = fmaf(s_a[w][c], carry, s_b[w][c]);
      }
    }
    __syncthreads();
    float s = s_in[grp][c];
#pragma unroll
    for (int i = 0; i < MG_TOK; i++) {
      const int t = t0 + grp * MG_TOK + i;
      s = fmaf(1.0f - z[i], s, u[i]);
      if (ok && t < Sc) out[((size_t)t * B + b) * ldo + ch] = from_f32<T>(s * silu_f32(g[i]));
    }
  }
  pdl_launch();
  if (grp == 0 && ok) *st = carry;
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
  return jg_launch(dev, "mingru_scan", mingru_scan_kernel<T>, dim3((unsigned)((d->width + MG_CH - 1) / MG_CH), (unsigned)b->B), dim3(MG_THREADS), 0, (const T*)d->proj, (float*)d->state,
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

// Portions, step 1: convolutions, unit vectors and gates into scratch.  A warp takes one q or k head, or a run of value
// channels, and walks DP_TOK consecutive tokens of a sequence with the taps and the last inputs in registers; the last unit
// is the gates.  NI * 32 channels per unit; TAPS = 0: any number of taps, inputs read again for every token.
constexpr int DP_TOK = 16;
template <typename T, int NI, int TAPS>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaArgs<T> a) {
  constexpr int KEEP = TAPS > 0 ? TAPS : 1;
  pdl_wait();
  const int lane = threadIdx.x & 31, C = a.channels(), nqk = 2 * a.G * a.dim, run = NI * 32;
  const int n_units = 2 * a.G + (a.H * a.vd + run - 1) / run + 1, unit = blockIdx.x * 8 + (threadIdx.x >> 5), b = blockIdx.z;
  const int s0 = blockIdx.y * DP_TOK, s1 = min(a.Sc, s0 + DP_TOK), p0 = a.pos[b];
  if (unit >= n_units) return;
  if (unit == n_units - 1) {
    for (int i = lane; i < (s1 - s0) * a.H; i += 32) {
      const size_t r = (size_t)(s0 + i / a.H) * a.B + b;
      *reinterpret_cast<float2*>(a.gates + (r * a.H + i % a.H) * 2) = delta_gates(a, r, i % a.H);
    }
    return;
  }
  const bool head = unit < 2 * a.G;  // q heads, then k heads, then value channels
  const int c0 = head ? unit * a.dim : nqk + (unit - 2 * a.G) * run, n = head ? a.dim : min(run, C - c0);
  const T* tail = a.tail + (size_t)a.seq[b] * a.taps * C;
  auto input = [&](int s, int c) -> float {  // token s of this call, or one before it
    if (s >= 0) return to_f32(a.proj[((size_t)s * a.B + b) * a.ldp + c]);
    return p0 + s >= 0 ? to_f32(tail[(size_t)((p0 + s) % a.taps) * C + c]) : 0.f;
  };
  float w[NI][KEEP], x[NI][KEEP];  // x[i][KEEP - 1]: the newest input
  if (TAPS > 0) {
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
      for (int j = 0; j < KEEP; j++) {
        const bool in = i * 32 + lane < n;
        w[i][j] = in ? a.conv_w[(size_t)(c0 + i * 32 + lane) * a.taps + j] : 0.f;
        x[i][j] = in && j > 0 ? input(s0 - KEEP + j, c0 + i * 32 + lane) : 0.f;
      }
  }
  T ahead[NI];
  auto fetch = [&](int s) {
#pragma unroll
    for (int i = 0; i < NI; i++)
      if (s < s1 && i * 32 + lane < n) ahead[i] = a.proj[((size_t)s * a.B + b) * a.ldp + c0 + i * 32 + lane];
  };
  if (TAPS > 0) fetch(s0);
  const float unit_scale = head && unit < a.G ? 1.0f / sqrtf((float)a.dim) : 1.0f;
  for (int s = s0; s < s1; s++) {
    float y[NI], ss = 0.f;
    if (TAPS > 0) {
#pragma unroll
      for (int i = 0; i < NI; i++) {
#pragma unroll
        for (int j = 0; j + 1 < KEEP; j++) x[i][j] = x[i][j + 1];
        x[i][KEEP - 1] = i * 32 + lane < n ? to_f32(ahead[i]) : 0.f;
      }
      fetch(s + 1);
    }
#pragma unroll
    for (int i = 0; i < NI; i++) {
      float acc = 0.f;
      if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < KEEP; j++) acc = fmaf(w[i][j], x[i][j], acc);
      } else if (i * 32 + lane < n) {
        const int c = c0 + i * 32 + lane;
        for (int j = 0; j < a.taps; j++) acc = fmaf(a.conv_w[(size_t)c * a.taps + j], input(s - (a.taps - 1 - j), c), acc);
      }
      y[i] = silu_f32(acc);
      ss = fmaf(y[i], y[i], ss);
    }
    const size_t r = (size_t)s * a.B + b;
    if (head) {
      const float rs = unit_scale / sqrtf(warp_sum(ss) + DELTA_UNIT_EPS);
      float* dst = a.qk + ((r * a.G + (unit < a.G ? unit : unit - a.G)) * 2 + (unit < a.G ? 0 : 1)) * a.lds;
#pragma unroll
      for (int i = 0; i < NI; i++)
        if (i * 32 + lane < a.lds) dst[i * 32 + lane] = i * 32 + lane < n ? y[i] * rs : 0.f;
    } else {
      float* dst = a.v + r * a.H * a.vd + c0 - nqk;
#pragma unroll
      for (int i = 0; i < NI; i++)
        if (i * 32 + lane < n) dst[i * 32 + lane] = y[i];
    }
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
// A lane holds E elements of each of four columns (so that a loaded piece of k or q serves four), 16 lanes a group of
// four columns; the partial sums are exchanged so that each lane ends up with one column's, solves that one, and hands the
// updates back to the group.
constexpr int DL_LPC = 8;  // lanes per column of the decode kernel below
constexpr int DS_LPC = 16, DS_NC = 4, DS_THREADS = 128, DS_COLS = DS_THREADS / DS_LPC * DS_NC, DS_TOK = 16, DS_STEP = 4, DS_PAIRS = DS_STEP * DS_STEP;

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
  constexpr int V = E < 4 ? 2 : 4;  // elements of a lane's contiguous pieces
  const int tid = threadIdx.x, l = tid % DS_LPC, h = blockIdx.y, b = blockIdx.z;
  // columns of the CTA: j0 ..; of this lane's group: jc .. jc + 3; the one this lane solves: j0 + col
  const int j0 = blockIdx.x * DS_COLS, jc = j0 + tid / DS_LPC * DS_NC, col = tid / DS_LPC * DS_NC + (l >> 2), g = h / (a.H / a.G), C = a.channels();
  for (int i = tid; i < (int)(2 * sizeof(Stage) / 4); i += DS_THREADS) reinterpret_cast<float*>(dsm)[i] = 0.f;  // padding, columns past vd
  __syncthreads();
  pdl_wait();
  const int slot = a.seq[b];
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
  // chunk e of a lane: V elements from (l + DS_LPC * e) * V on
  const bool cont = a.pos[b] > 0;
  float2 S[DS_NC][E / 2];
#pragma unroll
  for (int c = 0; c < DS_NC; c++) {
    const float* sp = a.state + (((size_t)slot * a.H + h) * a.vd + min(jc + c, a.vd - 1)) * a.lds;
#pragma unroll
    for (int e = 0; e < E / 2; e++) {
      const int off = (l + DS_LPC * (2 * e / V)) * V + 2 * e % V;
      S[c][e] = (cont && jc + c < a.vd && off < a.lds) ? *reinterpret_cast<const float2*>(sp + off) : make_float2(0.f, 0.f);
    }
  }

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
      float sk[DS_NC][DS_STEP], sq[DS_NC][DS_STEP];
      float2 kr[DS_STEP][E / 2];
#pragma unroll
      for (int i = 0; i < DS_STEP; i++) {
        float2 qr[E / 2];
#pragma unroll
        for (int e = 0; e < E / V; e++) {
          const float *kp = &st.k[tb + i][(l + DS_LPC * e) * V], *qp = &st.q[tb + i][(l + DS_LPC * e) * V];
          if constexpr (V == 4) {
            const float4 kv = *reinterpret_cast<const float4*>(kp), qv = *reinterpret_cast<const float4*>(qp);
            kr[i][2 * e] = make_float2(kv.x, kv.y); kr[i][2 * e + 1] = make_float2(kv.z, kv.w);
            qr[2 * e] = make_float2(qv.x, qv.y); qr[2 * e + 1] = make_float2(qv.z, qv.w);
          } else {
            kr[i][e] = *reinterpret_cast<const float2*>(kp);
            qr[e] = *reinterpret_cast<const float2*>(qp);
          }
        }
#pragma unroll
        for (int c = 0; c < DS_NC; c++) {
          float2 ak = make_float2(0.f, 0.f), aq = make_float2(0.f, 0.f);
#pragma unroll
          for (int e = 0; e < E / 2; e++) { ak = fma2(S[c][e], kr[i][e], ak); aq = fma2(S[c][e], qr[e], aq); }
          sk[c][i] = ak.x + ak.y;
          sq[c][i] = aq.x + aq.y;
        }
      }
      // exchange: lanes with bit 3 keep columns 2 and 3, then those with bit 2 the upper of their two; then all-reduce over 4
      const bool up8 = l & 8, up4 = l & 4;
      float mk[DS_STEP], mq[DS_STEP];
#pragma unroll
      for (int i = 0; i < DS_STEP; i++) {
        float k2[2], q2[2];
#pragma unroll
        for (int c = 0; c < 2; c++) {
          k2[c] = (up8 ? sk[c + 2][i] : sk[c][i]) + __shfl_xor_sync(0xffffffffu, up8 ? sk[c][i] : sk[c + 2][i], 8);
          q2[c] = (up8 ? sq[c + 2][i] : sq[c][i]) + __shfl_xor_sync(0xffffffffu, up8 ? sq[c][i] : sq[c + 2][i], 8);
        }
        mk[i] = (up4 ? k2[1] : k2[0]) + __shfl_xor_sync(0xffffffffu, up4 ? k2[0] : k2[1], 4);
        mq[i] = (up4 ? q2[1] : q2[0]) + __shfl_xor_sync(0xffffffffu, up4 ? q2[0] : q2[1], 4);
      }
#pragma unroll
      for (int o = 2; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < DS_STEP; i++) { mk[i] += __shfl_xor_sync(0xffffffffu, mk[i], o); mq[i] += __shfl_xor_sync(0xffffffffu, mq[i], o); }
      float w[DS_STEP], D = 1.f, mine = 0.f;
#pragma unroll
      for (int i = 0; i < DS_STEP; i++) {
        const float2 gt = *reinterpret_cast<const float2*>(st.gate[tb + i]);
        D *= gt.x;
        float pre = D * mk[i], o = D * mq[i];
#pragma unroll
        for (int jj = 0; jj < i; jj++) {
          w[jj] *= gt.x;
          pre = fmaf(pairs[grp][0][i * DS_STEP + jj], w[jj], pre);
          o = fmaf(pairs[grp][1][i * DS_STEP + jj], w[jj], o);
        }
        w[i] = gt.y * (st.v[tb + i][col] - pre);
        o = fmaf(pairs[grp][1][i * DS_STEP + i], w[i], o);
        if ((l & 3) == i) mine = o;
      }
      const float2 D2 = make_float2(D, D);
#pragma unroll
      for (int c = 0; c < DS_NC; c++) {
#pragma unroll
        for (int e = 0; e < E / 2; e++) S[c][e] = mul2(S[c][e], D2);
#pragma unroll
        for (int i = 0; i < DS_STEP; i++) {
          const float wc = __shfl_sync(0xffffffffu, w[i], c * 4, DS_LPC);
          const float2 w2 = make_float2(wc, wc);
#pragma unroll
          for (int e = 0; e < E / 2; e++) S[c][e] = fma2(kr[i][e], w2, S[c][e]);
        }
      }
      const int t = t0 + tb + (l & 3);
      if (j0 + col < a.vd && t < a.Sc) a.o[((size_t)t * a.B + b) * a.H * a.vd + (size_t)h * a.vd + j0 + col] = mine;
    }
    __syncthreads();  // the other stage is refilled next, and `pairs` is rewritten
  }
  pdl_launch();
#pragma unroll
  for (int c = 0; c < DS_NC; c++) {
    if (jc + c >= a.vd) continue;
    float* sp = a.state + (((size_t)slot * a.H + h) * a.vd + jc + c) * a.lds;
#pragma unroll
    for (int e = 0; e < E / 2; e++) {
      const int off = (l + DS_LPC * (2 * e / V)) * V + 2 * e % V;
      if (off < a.lds) *reinterpret_cast<float2*>(sp + off) = S[c][e];
    }
  }
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
constexpr int DD_THREADS = 256, DD_COLS = DD_THREADS / DL_LPC, DD_MAX_CLUSTER = 8;

template <typename T, int E>
__global__ void __launch_bounds__(DD_THREADS) delta_step_kernel(const DeltaArgs<T> a) {
  constexpr int DP = E * DL_LPC;
  extern __shared__ __align__(16) float dyn[];  // this CTA's columns: v, then o
  __shared__ __align__(16) float sk[DP], sq[DP];
  __shared__ float red[3][DD_THREADS / 32], s_ss[DD_MAX_CLUSTER];
  cg::cluster_group cluster = cg::this_cluster();
  const int cr = (int)cluster.block_rank(), cs = (int)cluster.num_blocks();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, l = tid % DL_LPC, col = tid / DL_LPC, h = blockIdx.y, r = blockIdx.z;
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
  DeltaCol<DL_LPC, E> S;
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
    k4[i] = *reinterpret_cast<const float4*>(&sk[(l + DL_LPC * i) * 4]);
    q4[i] = *reinterpret_cast<const float4*>(&sq[(l + DL_LPC * i) * 4]);
    k4[i].x *= rk; k4[i].y *= rk; k4[i].z *= rk; k4[i].w *= rk;
    q4[i].x *= rq; q4[i].y *= rq; q4[i].z *= rq; q4[i].w *= rq;
  }
  float ss = 0.f;
  for (int jb = j0; jb < j1; jb += DD_COLS) {  // the whole warp takes part in the shuffles
    const int j = jb + col;
    const bool live = j < j1;
    float* st = st0 + (size_t)(live ? j : j0) * a.lds;
    DeltaCol<DL_LPC, E> next;
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

template <typename T, int DP>  // DP: head size rounded up to 32, 64, 128 or 256
static int delta_launch(jg_dev* dev, const DeltaArgs<T>& a) {
  const int R = a.B * a.Sc;
  if (a.Sc == 1) {
    int cs = 1;
    while (cs < DD_MAX_CLUSTER && cs * DD_COLS < a.vd && R * a.H * cs < 2 * dev->sm_count) cs *= 2;
    const size_t smem = (size_t)((a.vd + cs - 1) / cs) * sizeof(float);
    return jg_launch_cluster(dev, "delta_step", delta_step_kernel<T, DP / DL_LPC>, dim3((unsigned)cs, (unsigned)a.H, (unsigned)R), dim3(DD_THREADS), smem, cs, a);
  }
  constexpr int E = DP / DS_LPC, NI = DP <= 128 ? 4 : 8;
  const dim3 pg((unsigned)((2 * a.G + (a.H * a.vd + NI * 32 - 1) / (NI * 32) + 1 + 7) / 8), (unsigned)((a.Sc + DP_TOK - 1) / DP_TOK), (unsigned)a.B);
  int rc = a.taps == 4 ? jg_launch(dev, "delta_prep", delta_prep_kernel<T, NI, 4>, pg, dim3(256), 0, a) : jg_launch(dev, "delta_prep", delta_prep_kernel<T, NI, 0>, pg, dim3(256), 0, a);
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
  if (d->dim <= 32) return delta_launch<T, 32>(dev, a);
  if (d->dim <= 64) return delta_launch<T, 64>(dev, a);
  if (d->dim <= 128) return delta_launch<T, 128>(dev, a);
  if (d->dim <= 256) return delta_launch<T, 256>(dev, a);
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
