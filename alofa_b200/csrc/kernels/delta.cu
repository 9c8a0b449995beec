// Two recurrences with a state of fixed size per request, both fp32 throughout and walked token by
// token in prompts and decoding alike, so that a position's value does not depend on how the
// prompt was cut or on what else is in the batch (the order of additions is fixed by the sizes).
//
// min_gru: element by element, S_t = (1 - z_t) S_(t-1) + z_t c_t with z = sigmoid(.), the candidate
//   c = x + 1/2 where x >= 0 and sigmoid(x) where x < 0; the output is S_t * silu(gate).
//
// The gated delta rule over a matrix state per head (N key channels x P value channels), with one
// decay per head and key channel, or one per head (g_t then is a number):
//   S <- diag(g_t) S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t
// so the read-out sees the token's own write.  A value channel's column of S never meets another
// column: o_t[p] = (g S[:, p]) . q + u[p] (k . q), and u[p] needs (g S[:, p]) . k.  Both dot
// products of the decayed column are taken in one round of exchanges between the threads that
// share the column; k . q comes ready from delta_prepare.
#include "common.cuh"

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ---------------------------------------------------------------------------
// min_gru: u [T, ld] fp32 holds the projections' sums (biases added) at columns z_off, x_off, g_off;
// out [T, width] in the compute dtype; state [slots][>= width] fp32.  A block takes 32 channels (a
// lane each) of one request; its warps share the request's tokens of the step, a stretch of
// consecutive tokens each.  The recurrence is linear in the state, so a stretch is the map
// S -> A S + B with A = prod (1 - z_t) and B its result from a zero state: every warp finds its
// stretch's (A, B), the stretches before it give its starting state (in order, from the request's
// stored state), and it then walks its stretch and writes the outputs.  A warp reads GRU_AHEAD
// tokens' inputs before it uses the first, so that the loads do not wait on one another.  Decode
// steps are launched with one warp a block, which walks its (one) token from the stored state.
// ---------------------------------------------------------------------------
constexpr int GRU_AHEAD = 8;
constexpr int GRU_MAX_WARPS = 16;

__device__ __forceinline__ float gru_candidate(float x) { return x >= 0.f ? x + 0.5f : sigmoid_f(x); }

template <typename TO>
__global__ void __launch_bounds__(GRU_MAX_WARPS * 32) min_gru_kernel(TO* __restrict__ out, const float* __restrict__ u, int ld, int z_off, int x_off, int g_off,
                                                                      float* __restrict__ state, long long slot_stride, const int* __restrict__ q_start,
                                                                      const int* __restrict__ state_slots, int width) {
  __shared__ float seg_a[GRU_MAX_WARPS][32], seg_b[GRU_MAX_WARPS][32];
  pdl_begin();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int c = blockIdx.x * 32 + lane, s = blockIdx.y;
  const bool live = c < width;
  const int t0 = q_start[s], t1 = q_start[s + 1];
  if (t0 >= t1) return;  // the whole block
  const int per = (t1 - t0 + warps - 1) / warps;
  const int a = min(t0 + warp * per, t1), b = min(a + per, t1);
  const float* col = u + (live ? c : 0);
  if (warps > 1) {
    float A = 1.f, B = 0.f;
    for (int t = a; t < b; t += GRU_AHEAD) {
      float zs[GRU_AHEAD], xs[GRU_AHEAD];
#pragma unroll
      for (int i = 0; i < GRU_AHEAD; ++i) {
        const float* row = col + (size_t)min(t + i, b - 1) * ld;
        zs[i] = row[z_off];
        xs[i] = row[x_off];
      }
#pragma unroll
      for (int i = 0; i < GRU_AHEAD; ++i) {
        if (t + i >= b) break;
        const float z = sigmoid_f(zs[i]);
        B = (1.0f - z) * B + z * gru_candidate(xs[i]);
        A *= 1.0f - z;
      }
    }
    seg_a[warp][lane] = A;
    seg_b[warp][lane] = B;
    __syncthreads();
  }
  if (a >= b || !live) return;
  float* st = state + (long long)state_slots[s] * slot_stride + c;
  float S = *st;
  for (int w = 0; w < warp; ++w) S = seg_a[w][lane] * S + seg_b[w][lane];
  for (int t = a; t < b; t += GRU_AHEAD) {
    float zs[GRU_AHEAD], xs[GRU_AHEAD], gs[GRU_AHEAD];
#pragma unroll
    for (int i = 0; i < GRU_AHEAD; ++i) {
      const float* row = col + (size_t)min(t + i, b - 1) * ld;
      zs[i] = row[z_off];
      xs[i] = row[x_off];
      gs[i] = row[g_off];
    }
#pragma unroll
    for (int i = 0; i < GRU_AHEAD; ++i) {
      if (t + i >= b) break;
      const float z = sigmoid_f(zs[i]);
      S = (1.0f - z) * S + z * gru_candidate(xs[i]);
      out[(size_t)(t + i) * width + c] = from_f<TO>(S * (gs[i] / (1.0f + expf(-gs[i]))));
    }
  }
  if (b == t1) *st = S;  // the stretch that ends the request's tokens leaves the state
}

// n_tokens: rows of the step.  With as many rows as requests every request has one token.
ALOFA_API int alofa_min_gru(void* out, const float* u, int ld, int z_off, int x_off, int g_off, float* state, long long slot_stride, const int* q_start,
                            const int* state_slots, int n_seqs, int n_tokens, int width, int out_bf16, cudaStream_t stream) {
  if (n_seqs <= 0) return ALOFA_OK;
  if (width <= 0) return ALOFA_ERR_ARGUMENT;
  const dim3 grid((width + 31) / 32, n_seqs);
  // stretches of 16 tokens or more: shorter ones cost more in the (A, B) pass than they save
  int warps = 1;
  while (warps < GRU_MAX_WARPS && (long long)n_tokens >= (long long)n_seqs * warps * 2 * 16) warps *= 2;
  if (out_bf16) launch_dep(min_gru_kernel<bf16>, grid, warps * 32, 0, stream, (bf16*)out, u, ld, z_off, x_off, g_off, state, slot_stride, q_start, state_slots, width);
  else launch_dep(min_gru_kernel<float>, grid, warps * 32, 0, stream, (float*)out, u, ld, z_off, x_off, g_off, state, slot_stride, q_start, state_slots, width);
  return launch_status();
}

// ---------------------------------------------------------------------------
// delta_prepare: what the recurrence reads, once per token.  conv [T, ldc] fp32 holds the
// convolved and activated [q: G * N | k: G * N | v: H * P]; dz [T, ldz] the decays' logits (H * N of them);
// u [T, ldu] the gate logit of each head at column b_off.
//   qn = q / sqrt(sum(q^2) + unit_eps) * q_scale,  kn = k / sqrt(sum(k^2) + unit_eps)   per group
//   kq[t, g] = kn . qn
//   g[t, h, n] = exp(-exp(A_log[h]) * softplus(dz[t, h, n] + dt_bias[h, n]))      (ND = N decays a head, or ND = 1: g[t, h])
//   beta[t, h] = sigmoid(u[t, b_off + h])
// One block per token, a warp per group in turn.
// ---------------------------------------------------------------------------
__global__ void __launch_bounds__(256) delta_prepare_kernel(float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ kq, float* __restrict__ g,
                                                            float* __restrict__ beta, const float* __restrict__ conv, int ldc, const float* __restrict__ dz, int ldz,
                                                            const float* __restrict__ u, int ldu, int b_off, const float* __restrict__ dt_bias,
                                                            const float* __restrict__ A_log, int H, int G, int N, int ND, float unit_eps, float q_scale) {
  pdl_begin();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
  const float* row = conv + (size_t)t * ldc;
  for (int grp = warp; grp < G; grp += nwarp) {
    const float* q = row + (size_t)grp * N;
    const float* k = row + (size_t)(G + grp) * N;
    float sq = 0.f, sk = 0.f;
    for (int n = lane; n < N; n += 32) {
      sq = fmaf(q[n], q[n], sq);
      sk = fmaf(k[n], k[n], sk);
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    const float rq = q_scale / sqrtf(sq + unit_eps), rk = 1.0f / sqrtf(sk + unit_eps);
    float dot = 0.f;
    for (int n = lane; n < N; n += 32) {
      const float a = q[n] * rq, b = k[n] * rk;
      qn[((size_t)t * G + grp) * N + n] = a;
      kn[((size_t)t * G + grp) * N + n] = b;
      dot = fmaf(a, b, dot);
    }
    dot = warp_sum(dot);
    if (lane == 0) kq[(size_t)t * G + grp] = dot;
  }
  for (int e = threadIdx.x; e < H * ND; e += blockDim.x) {
    const int h = e / ND;
    g[(size_t)t * H * ND + e] = expf(-expf(A_log[h]) * softplus_f(dz[(size_t)t * ldz + e] + dt_bias[e]));
  }
  for (int h = threadIdx.x; h < H; h += blockDim.x) beta[(size_t)t * H + h] = sigmoid_f(u[(size_t)t * ldu + b_off + h]);
}

ALOFA_API int alofa_delta_prepare(float* qn, float* kn, float* kq, float* g, float* beta, const float* conv, int ldc, const float* dz, int ldz, const float* u, int ldu,
                                  int b_off, const float* dt_bias, const float* A_log, int n_tokens, int H, int G, int N, int ND, float unit_eps, float q_scale,
                                  cudaStream_t stream) {
  if (n_tokens <= 0) return ALOFA_OK;
  if (H <= 0 || G <= 0 || H % G || N <= 0 || (ND != N && ND != 1)) return ALOFA_ERR_ARGUMENT;
  launch_dep(delta_prepare_kernel, n_tokens, 256, 0, stream, qn, kn, kq, g, beta, conv, ldc, dz, ldz, u, ldu, b_off, dt_bias, A_log, H, G, N, ND, unit_eps, q_scale);
  return launch_status();
}

// ---------------------------------------------------------------------------
// delta_scan: a block takes one (head, request) and PC value channels and walks the request's
// tokens of the step in order.  The NS threads that share a value channel (neighbours in a warp)
// each hold R key channels of its column in registers, four neighbours at a time: channels 4 ns ..
// 4 ns + 3, then those 4 NS further on, ... (a token's keys, queries and decays are then R / 4 loads of
// 16 bytes each, and the NS threads' loads lie side by side in shared memory).  The state lies
// in memory as [head][value channel][key channel].  Keys, queries, decays, values, beta and k . q
// of TC tokens at a time come into shared memory by asynchronous copies, the next ones while
// these are worked on.  ONE: one decay per head: it travels beside beta and k . q and multiplies the column.
// ---------------------------------------------------------------------------
struct DeltaArgs {
  float* y;                              // [T, H * P]
  const float* v; int ldv, v_off;        // values: v[t * ldv + v_off + h * P + p]
  const float* kn; const float* qn;      // [T, G, N]
  const float* kq;                       // [T, G]
  const float* g;                        // [T, H, N], ONE: [T, H]
  const float* beta;                     // [T, H]
  float* state; long long slot_stride;
  const int* q_start; const int* state_slots;
  int H, G, N, P, NS, PC, TC, vec;
};

__device__ __forceinline__ void delta_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void delta_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void delta_cp_done() {
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

template <int R, bool ONE>
__global__ void __launch_bounds__(256) delta_scan_kernel(const DeltaArgs a) {
  extern __shared__ __align__(16) float delta_smem[];
  const int N = a.N, P = a.P, NS = a.NS, PC = a.PC, TC = a.TC;
  const int NW = NS * R;                       // key channels a stage holds per token (zeros past N)
  const int per_stage = TC * ((ONE ? 2 : 3) * NW + PC + 4);  // k, q, g (unless ONE), v, then beta, k.q and (ONE) the decay (padded to four words)
  const int h = blockIdx.x, s = blockIdx.y, p0 = blockIdx.z * PC;
  const int tid = threadIdx.x, nthreads = blockDim.x;
  const int pl = tid / NS, ns = tid - pl * NS;
  const int p = p0 + pl;
  const bool live_p = pl < PC && p < P;
  const int grp = h / (a.H / a.G);
  for (int e = tid; e < 2 * per_stage; e += nthreads) delta_smem[e] = 0.f;  // the rows' tails that no copy writes stay zero
  pdl_begin();
  const int t0 = a.q_start[s], t1 = a.q_start[s + 1];
  float* S = a.state + (long long)a.state_slots[s] * a.slot_stride + ((size_t)h * P + (live_p ? p : 0)) * N;
  float st[R];
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int n = (j >> 2) * 4 * NS + 4 * ns + (j & 3);
    st[j] = (live_p && n < N) ? S[n] : 0.f;
  }
  __syncthreads();

  auto fetch = [&](int which, int c0) {
    float* ks = delta_smem + which * per_stage;
    float* qs = ks + TC * NW;
    float* gs = qs + TC * NW;
    float* vs = ONE ? gs : gs + TC * NW;
    float* bs = vs + TC * PC;
    const int live = min(TC, t1 - c0);
    if (a.vec) {
      const int n4 = N >> 2;
      for (int e = tid; e < live * n4; e += nthreads) {
        const int tt = e / n4, c = (e - tt * n4) * 4;
        const size_t t = c0 + tt;
        delta_cp16(ks + tt * NW + c, a.kn + (t * a.G + grp) * N + c);
        delta_cp16(qs + tt * NW + c, a.qn + (t * a.G + grp) * N + c);
        if (!ONE) delta_cp16(gs + tt * NW + c, a.g + (t * a.H + h) * N + c);
      }
      const int p4 = PC >> 2;
      for (int e = tid; e < live * p4; e += nthreads) {
        const int tt = e / p4, c = (e - tt * p4) * 4;
        if (p0 + c < P) delta_cp16(vs + tt * PC + c, a.v + (size_t)(c0 + tt) * a.ldv + a.v_off + h * P + p0 + c);
      }
    } else {
      for (int e = tid; e < live * N; e += nthreads) {
        const int tt = e / N, c = e - tt * N;
        const size_t t = c0 + tt;
        delta_cp4(ks + tt * NW + c, a.kn + (t * a.G + grp) * N + c);
        delta_cp4(qs + tt * NW + c, a.qn + (t * a.G + grp) * N + c);
        if (!ONE) delta_cp4(gs + tt * NW + c, a.g + (t * a.H + h) * N + c);
      }
      for (int e = tid; e < live * PC; e += nthreads) {
        const int tt = e / PC, c = e - tt * PC;
        if (p0 + c < P) delta_cp4(vs + tt * PC + c, a.v + (size_t)(c0 + tt) * a.ldv + a.v_off + h * P + p0 + c);
      }
    }
    for (int tt = tid; tt < live; tt += nthreads) {
      delta_cp4(bs + 4 * tt, a.beta + (size_t)(c0 + tt) * a.H + h);
      delta_cp4(bs + 4 * tt + 1, a.kq + (size_t)(c0 + tt) * a.G + grp);
      if (ONE) delta_cp4(bs + 4 * tt + 2, a.g + (size_t)(c0 + tt) * a.H + h);
    }
  };

  if (t0 < t1) fetch(0, t0);
  int which = 0;
  for (int c0 = t0; c0 < t1; c0 += TC, which ^= 1) {
    delta_cp_done();
    __syncthreads();  // this stage has arrived for everyone, and everyone is done with the other
    if (c0 + TC < t1) fetch(which ^ 1, c0 + TC);
    const int live = min(TC, t1 - c0);
    const float* ks = delta_smem + which * per_stage;
    const float* qs = ks + TC * NW;
    const float* gs = qs + TC * NW;
    const float* vs = ONE ? gs : gs + TC * NW;
    const float* bs = vs + TC * PC;
    for (int tt = 0; tt < live; ++tt) {
      const float4* kr = reinterpret_cast<const float4*>(ks + tt * NW) + ns;
      const float4* qr = reinterpret_cast<const float4*>(qs + tt * NW) + ns;
      const float4* gr = reinterpret_cast<const float4*>(gs + tt * NW) + ns;
      const float decay = ONE ? bs[4 * tt + 2] : 0.f;
      float kk[R];
      float r0 = 0.f, r1 = 0.f, w0 = 0.f, w1 = 0.f;
#pragma unroll
      for (int j4 = 0; j4 < R / 4; ++j4) {
        const float4 k4 = kr[j4 * NS], q4 = qr[j4 * NS], g4 = ONE ? make_float4(decay, decay, decay, decay) : gr[j4 * NS];
        const int j = 4 * j4;
        kk[j] = k4.x, kk[j + 1] = k4.y, kk[j + 2] = k4.z, kk[j + 3] = k4.w;
        st[j] *= g4.x, st[j + 1] *= g4.y, st[j + 2] *= g4.z, st[j + 3] *= g4.w;
        r0 = fmaf(st[j], k4.x, r0);
        w0 = fmaf(st[j], q4.x, w0);
        r1 = fmaf(st[j + 1], k4.y, r1);
        w1 = fmaf(st[j + 1], q4.y, w1);
        r0 = fmaf(st[j + 2], k4.z, r0);
        w0 = fmaf(st[j + 2], q4.z, w0);
        r1 = fmaf(st[j + 3], k4.w, r1);
        w1 = fmaf(st[j + 3], q4.w, w1);
      }
      float r = r0 + r1, w = w0 + w1;
      for (int o = NS >> 1; o > 0; o >>= 1) {
        r += __shfl_xor_sync(0xffffffffu, r, o);
        w += __shfl_xor_sync(0xffffffffu, w, o);
      }
      const float vv = pl < PC ? vs[tt * PC + pl] : 0.f;
      const float uu = bs[4 * tt] * (vv - r);
#pragma unroll
      for (int j = 0; j < R; ++j) st[j] = fmaf(kk[j], uu, st[j]);
      if (ns == 0 && live_p) a.y[(size_t)(c0 + tt) * a.H * P + h * P + p] = fmaf(uu, bs[4 * tt + 1], w);
    }
  }
  if (live_p && t0 < t1) {
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int n = (j >> 2) * 4 * NS + 4 * ns + (j & 3);
      if (n < N) S[n] = st[j];
    }
  }
}

template <int R, bool ONE>
static int delta_scan_launch(const DeltaArgs& a, int n_seqs, int threads, size_t smem, cudaStream_t stream) {
  static size_t set = 48 * 1024;
  if (smem > set) {
    if (cudaFuncSetAttribute(delta_scan_kernel<R, ONE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return ALOFA_ERR_LAUNCH;
    set = smem;
  }
  launch_dep(delta_scan_kernel<R, ONE>, dim3(a.H, n_seqs, (a.P + a.PC - 1) / a.PC), threads, smem, stream, a);
  return launch_status();
}

// one_decay: g is [T, H], one decay per head.  spread: how many blocks the scan should have at least, if the value channels allow it.
ALOFA_API int alofa_delta_scan(float* y, const float* v, int ldv, int v_off, const float* kn, const float* qn, const float* kq, const float* g, const float* beta,
                               float* state, long long slot_stride, const int* q_start, const int* state_slots, int n_tokens, int n_seqs, int H, int G, int N, int P,
                               int one_decay, int spread, cudaStream_t stream) {
  if (n_seqs <= 0 || n_tokens <= 0) return ALOFA_OK;
  if (H <= 0 || G <= 0 || H % G || N <= 0 || N > 1024 || P <= 0) return ALOFA_ERR_ARGUMENT;
  int R = N <= 64 ? 8 : (N <= 256 ? 16 : 32);
  // Prompt portions of few requests and heads wait on each token's chain of dependent instructions, not on
  // throughput: half the channels a thread (twice the threads to a value channel, one more level of exchange)
  // shortens it (4 heads of 128 x 256, one request of 2,048 tokens: 717 -> 610 us).  With blocks of 16 value
  // channels enough to fill the device it does not pay (8 such heads: the prompt step 4.06 -> 4.28 ms).
  if (R == 16 && N <= 128 && n_tokens >= 8 * n_seqs && (long long)H * n_seqs * ((P + 15) / 16) < spread) R = 8;
  int NS = 1;
  while (NS * R < N) NS *= 2;
  if (NS > 32) return ALOFA_ERR_ARGUMENT;
  int PC = 256 / NS;  // value channels per block, one per group of NS threads
  while (PC > 4 && PC / 2 >= P) PC /= 2;
  while (PC > 4 && PC * NS > 32 && (long long)H * n_seqs * ((P + PC - 1) / PC) < spread) PC /= 2;
  while (PC * NS < 32) PC *= 2;
  if (PC < 4) PC = 4;
  const int threads = (PC * NS + 31) / 32 * 32;
  const bool vec = N % 4 == 0 && P % 4 == 0 && PC % 4 == 0 && ldv % 4 == 0 && v_off % 4 == 0 && ((uintptr_t)v % 16 == 0) && ((uintptr_t)kn % 16 == 0) &&
                   ((uintptr_t)qn % 16 == 0) && (one_decay || (uintptr_t)g % 16 == 0);
  int TC = 16;
  const int wide = one_decay ? 2 : 3;  // rows of N numbers a token brings
  while (TC > 2 && (size_t)2 * TC * (wide * NS * R + PC + 4) * sizeof(float) > 160 * 1024) TC /= 2;
  const size_t smem = (size_t)2 * TC * (wide * NS * R + PC + 4) * sizeof(float);
  if (smem > 200 * 1024) return ALOFA_ERR_ARGUMENT;
  DeltaArgs a = {y, v, ldv, v_off, kn, qn, kq, g, beta, state, slot_stride, q_start, state_slots, H, G, N, P, NS, PC, TC, vec ? 1 : 0};
  if (one_decay) {
    if (R == 8) return delta_scan_launch<8, true>(a, n_seqs, threads, smem, stream);
    if (R == 16) return delta_scan_launch<16, true>(a, n_seqs, threads, smem, stream);
    return delta_scan_launch<32, true>(a, n_seqs, threads, smem, stream);
  }
  if (R == 8) return delta_scan_launch<8, false>(a, n_seqs, threads, smem, stream);
  if (R == 16) return delta_scan_launch<16, false>(a, n_seqs, threads, smem, stream);
  return delta_scan_launch<32, false>(a, n_seqs, threads, smem, stream);
}

// ---------------------------------------------------------------------------
// One decay per head, over portions of prompts: GROUP tokens at a time.  With a number for a decay the state a token meets is
// the one the group began with, decayed, plus the group's own writes before it, so that with S the state before the group,
// G_i = g_1 ... g_i and D_ij = g_(j+1) ... g_i (products, no quotients)
//   u_i = beta_i (v_i - G_i (S^T k_i) - sum_{j<i} D_ij (k_j . k_i) u_j)
//   o_i = G_i (S^T q_i) + sum_{j<=i} D_ij (k_j . q_i) u_j
//   S <- G_last S + sum_j D_last,j k_j u_j^T
// The 2 GROUP dot products with S are independent: their exchanges between the threads of a value channel run side by side
// once a group instead of one after the other every token, and the state is decayed once.  The products D_ij (k_j . k_i) and
// D_ij (k_j . q_i) of a token with the GROUP - 1 before it do not depend on where groups begin: delta_pairs makes them once for
// all value channels.  A group that a request's tokens of the step do not fill is filled with tokens of zeros and decay one.
// ---------------------------------------------------------------------------
constexpr int GROUP = 4;
constexpr int PAIR_WORDS = 12;  // beta, g, D (k_(t-d) . k_t) for d = 1 .. 3, D (k_(t-d) . q_t) for d = 0 .. 3, padding

__global__ void __launch_bounds__(256) delta_pairs_kernel(float* __restrict__ pairs, const float* __restrict__ kn, const float* __restrict__ qn, const float* __restrict__ kq,
                                                          const float* __restrict__ g, const float* __restrict__ beta, int n_tokens, int H, int G, int N) {
  pdl_begin();
  const int lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);  // a warp per (token, group)
  if (unit >= (long long)n_tokens * G) return;
  const int t = (int)(unit / G), grp = (int)(unit - (long long)t * G);
  float kk[GROUP - 1], qk[GROUP - 1];
#pragma unroll
  for (int d = 0; d < GROUP - 1; ++d) kk[d] = qk[d] = 0.f;
  const float* k0 = kn + ((size_t)t * G + grp) * N;
  const float* q0 = qn + ((size_t)t * G + grp) * N;
  const size_t row = (size_t)G * N;
  for (int n = lane; n < N; n += 32) {
    const float k = k0[n], q = q0[n];
#pragma unroll
    for (int d = 0; d < GROUP - 1; ++d) {
      const float before = t > d ? k0[n - (long long)(d + 1) * (long long)row] : 0.f;
      kk[d] = fmaf(before, k, kk[d]);
      qk[d] = fmaf(before, q, qk[d]);
    }
  }
#pragma unroll
  for (int d = 0; d < GROUP - 1; ++d) {
    kk[d] = warp_sum(kk[d]);
    qk[d] = warp_sum(qk[d]);
  }
  const int hg = H / G;
  for (int i = lane; i < hg; i += 32) {
    const int h = grp * hg + i;
    float* out = pairs + ((size_t)t * H + h) * PAIR_WORDS;
    out[0] = beta[(size_t)t * H + h];
    out[1] = g[(size_t)t * H + h];
    out[2 + GROUP - 1] = kq[(size_t)t * G + grp];
    float decay = 1.f;
#pragma unroll
    for (int d = 0; d < GROUP - 1; ++d) {
      decay *= t >= d ? g[(size_t)(t - d) * H + h] : 0.f;
      out[2 + d] = decay * kk[d];
      out[2 + GROUP + d] = decay * qk[d];
    }
#pragma unroll
    for (int e = 2 * GROUP + 1; e < PAIR_WORDS; ++e) out[e] = 0.f;
  }
}

ALOFA_API int alofa_delta_pair_words() { return PAIR_WORDS; }

// pairs [T, H, PAIR_WORDS]: what the grouped scan reads of a token beside its key, query and values.  kq [T, G], g and beta [T, H].
ALOFA_API int alofa_delta_pairs(float* pairs, const float* kn, const float* qn, const float* kq, const float* g, const float* beta, int n_tokens, int H, int G, int N,
                                cudaStream_t stream) {
  if (n_tokens <= 0) return ALOFA_OK;
  if (H <= 0 || G <= 0 || H % G || N <= 0 || (uintptr_t)pairs % 16) return ALOFA_ERR_ARGUMENT;
  const long long units = (long long)n_tokens * G;
  launch_dep(delta_pairs_kernel, (unsigned)((units + 7) / 8), 256, 0, stream, pairs, kn, qn, kq, g, beta, n_tokens, H, G, N);
  return launch_status();
}

// Sums of `a` over the NS neighbouring lanes that share a value channel (NS a power of two): every lane gets all of them.
template <int COUNT>
__device__ __forceinline__ void sum_over_lanes(float (&a)[COUNT], int NS, int lane) {
  static_assert(COUNT == 8, "three halving levels");
  if (NS < 8) {
    for (int o = NS >> 1; o > 0; o >>= 1) {
#pragma unroll
      for (int i = 0; i < COUNT; ++i) a[i] += __shfl_xor_sync(0xffffffffu, a[i], o);
    }
    return;
  }
  // three levels in which a lane hands half of its sums over and keeps the other half, then one sum a lane to the end, then everyone
  // fetches the sums from the lanes that hold them: sixteen exchanges and less instead of 8 log2 NS
#pragma unroll
  for (int level = 0, width = COUNT / 2; level < 3; ++level, width >>= 1) {
    const int o = NS >> (level + 1);
    const bool upper = lane & o;
#pragma unroll
    for (int i = 0; i < COUNT / 2; ++i) {
      if (i < width) {
        const float give = upper ? a[i] : a[i + width], keep = upper ? a[i + width] : a[i];
        a[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
      }
    }
  }
  float one = a[0];
  for (int o = NS >> 4; o > 0; o >>= 1) one += __shfl_xor_sync(0xffffffffu, one, o);
  const int base = lane & ~(NS - 1);
#pragma unroll
  for (int i = 0; i < COUNT; ++i) a[i] = __shfl_sync(0xffffffffu, one, base + ((i >> 2) & 1) * (NS >> 1) + ((i >> 1) & 1) * (NS >> 2) + (i & 1) * (NS >> 3));
}

struct DeltaGroupArgs {
  float* y;                              // [T, H * P]
  const float* v; int ldv, v_off;        // values: v[t * ldv + v_off + h * P + p]
  const float* kn; const float* qn;      // [T, G, N]
  const float* pairs;                    // [T, H, PAIR_WORDS]
  float* state; long long slot_stride;
  const int* q_start; const int* state_slots;
  int H, G, N, P, NS, PC, TC, vec;
};

// The block, its threads and their channels as in delta_scan_kernel; TC is a multiple of GROUP.
template <int R>
__global__ void __launch_bounds__(256) delta_group_scan_kernel(const DeltaGroupArgs a) {
  extern __shared__ __align__(16) float delta_smem[];
  const int N = a.N, P = a.P, NS = a.NS, PC = a.PC, TC = a.TC;
  const int NW = NS * R;
  const int per_stage = TC * (2 * NW + PC + PAIR_WORDS);  // k, q, v, the pair words
  const int h = blockIdx.x, s = blockIdx.y, p0 = blockIdx.z * PC;
  const int tid = threadIdx.x, nthreads = blockDim.x, lane = tid & 31;
  const int pl = tid / NS, ns = tid - pl * NS;
  const int p = p0 + pl;
  const bool live_p = pl < PC && p < P;
  const int grp = h / (a.H / a.G);
  for (int e = tid; e < 2 * per_stage; e += nthreads) delta_smem[e] = 0.f;  // the rows' tails that no copy writes stay zero
  pdl_begin();
  const int t0 = a.q_start[s], t1 = a.q_start[s + 1];
  float* S = a.state + (long long)a.state_slots[s] * a.slot_stride + ((size_t)h * P + (live_p ? p : 0)) * N;
  float st[R];
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int n = (j >> 2) * 4 * NS + 4 * ns + (j & 3);
    st[j] = (live_p && n < N) ? S[n] : 0.f;
  }
  __syncthreads();

  auto fetch = [&](int which, int c0) {
    float* ks = delta_smem + which * per_stage;
    float* qs = ks + TC * NW;
    float* ps = qs + TC * NW;
    float* vs = ps + TC * PAIR_WORDS;
    const int live = min(TC, t1 - c0);
    if (a.vec) {
      const int n4 = N >> 2, p4 = PC >> 2;
      for (int e = tid; e < live * n4; e += nthreads) {
        const int tt = e / n4, c = (e - tt * n4) * 4;
        const size_t at = ((size_t)(c0 + tt) * a.G + grp) * N + c;
        delta_cp16(ks + tt * NW + c, a.kn + at);
        delta_cp16(qs + tt * NW + c, a.qn + at);
      }
      for (int e = tid; e < live * p4; e += nthreads) {
        const int tt = e / p4, c = (e - tt * p4) * 4;
        if (p0 + c < P) delta_cp16(vs + tt * PC + c, a.v + (size_t)(c0 + tt) * a.ldv + a.v_off + h * P + p0 + c);
      }
    } else {
      for (int e = tid; e < live * N; e += nthreads) {
        const int tt = e / N, c = e - tt * N;
        const size_t at = ((size_t)(c0 + tt) * a.G + grp) * N + c;
        delta_cp4(ks + tt * NW + c, a.kn + at);
        delta_cp4(qs + tt * NW + c, a.qn + at);
      }
      for (int e = tid; e < live * PC; e += nthreads) {
        const int tt = e / PC, c = e - tt * PC;
        if (p0 + c < P) delta_cp4(vs + tt * PC + c, a.v + (size_t)(c0 + tt) * a.ldv + a.v_off + h * P + p0 + c);
      }
    }
    for (int e = tid; e < live * (PAIR_WORDS / 4); e += nthreads) {
      const int tt = e / (PAIR_WORDS / 4), c = (e - tt * (PAIR_WORDS / 4)) * 4;
      delta_cp16(ps + tt * PAIR_WORDS + c, a.pairs + ((size_t)(c0 + tt) * a.H + h) * PAIR_WORDS + c);
    }
    // the tokens that fill the last group up: zeros, and a decay of one
    for (int tt = live + tid; tt < (live + GROUP - 1) / GROUP * GROUP; tt += nthreads) {
      for (int c = 0; c < NW; ++c) ks[tt * NW + c] = qs[tt * NW + c] = 0.f;
      for (int c = 0; c < PC; ++c) vs[tt * PC + c] = 0.f;
      for (int c = 0; c < PAIR_WORDS; ++c) ps[tt * PAIR_WORDS + c] = c == 1 ? 1.f : 0.f;
    }
  };

  if (t0 < t1) fetch(0, t0);
  int which = 0;
  for (int c0 = t0; c0 < t1; c0 += TC, which ^= 1) {
    delta_cp_done();
    __syncthreads();  // this stage has arrived for everyone, and everyone is done with the other
    if (c0 + TC < t1) fetch(which ^ 1, c0 + TC);
    const int live = min(TC, t1 - c0);
    const float* ks = delta_smem + which * per_stage;
    const float* qs = ks + TC * NW;
    const float* ps = qs + TC * NW;
    const float* vs = ps + TC * PAIR_WORDS;
    for (int b = 0; b < live; b += GROUP) {
      float dot[2 * GROUP];  // S^T k_i, then S^T q_i
#pragma unroll
      for (int i = 0; i < GROUP; ++i) {
        const float4* kr = reinterpret_cast<const float4*>(ks + (b + i) * NW) + ns;
        const float4* qr = reinterpret_cast<const float4*>(qs + (b + i) * NW) + ns;
        float r = 0.f, w = 0.f;
#pragma unroll
        for (int j4 = 0; j4 < R / 4; ++j4) {
          const float4 k4 = kr[j4 * NS], q4 = qr[j4 * NS];
          const int j = 4 * j4;
          r = fmaf(st[j], k4.x, r);
          w = fmaf(st[j], q4.x, w);
          r = fmaf(st[j + 1], k4.y, r);
          w = fmaf(st[j + 1], q4.y, w);
          r = fmaf(st[j + 2], k4.z, r);
          w = fmaf(st[j + 2], q4.z, w);
          r = fmaf(st[j + 3], k4.w, r);
          w = fmaf(st[j + 3], q4.w, w);
        }
        dot[i] = r;
        dot[GROUP + i] = w;
      }
      sum_over_lanes<2 * GROUP>(dot, NS, lane);
      float u[GROUP], decay[GROUP];
      float so_far = 1.f;
#pragma unroll
      for (int i = 0; i < GROUP; ++i) {
        const float4* pr = reinterpret_cast<const float4*>(ps + (b + i) * PAIR_WORDS);
        const float4 pa = pr[0], pb = pr[1];  // beta, g, kk1, kk2 | kk3, qk0, qk1, qk2
        const float qk3 = ps[(b + i) * PAIR_WORDS + 8];
        const float kk[GROUP - 1] = {pa.z, pa.w, pb.x}, qk[GROUP] = {pb.y, pb.z, pb.w, qk3};
        decay[i] = pa.y;
        so_far *= pa.y;
        float x = (pl < PC ? vs[(b + i) * PC + pl] : 0.f) - so_far * dot[i];
        float o = so_far * dot[GROUP + i];
#pragma unroll
        for (int j = 0; j < GROUP; ++j)
          if (j < i) {
            x = fmaf(-kk[i - j - 1], u[j], x);
            o = fmaf(qk[i - j], u[j], o);
          }
        u[i] = pa.x * x;
        o = fmaf(qk[0], u[i], o);
        if (ns == 0 && live_p && b + i < live) a.y[(size_t)(c0 + b + i) * a.H * P + h * P + p] = o;
      }
      float later = 1.f;  // the decays after token i
#pragma unroll
      for (int i = GROUP - 1; i >= 0; --i) {
        u[i] *= later;
        later *= decay[i];
      }
#pragma unroll
      for (int j = 0; j < R; ++j) st[j] *= so_far;
#pragma unroll
      for (int i = 0; i < GROUP; ++i) {
        const float4* kr = reinterpret_cast<const float4*>(ks + (b + i) * NW) + ns;
#pragma unroll
        for (int j4 = 0; j4 < R / 4; ++j4) {
          const float4 k4 = kr[j4 * NS];
          const int j = 4 * j4;
          st[j] = fmaf(k4.x, u[i], st[j]);
          st[j + 1] = fmaf(k4.y, u[i], st[j + 1]);
          st[j + 2] = fmaf(k4.z, u[i], st[j + 2]);
          st[j + 3] = fmaf(k4.w, u[i], st[j + 3]);
        }
      }
    }
  }
  if (live_p && t0 < t1) {
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int n = (j >> 2) * 4 * NS + 4 * ns + (j & 3);
      if (n < N) S[n] = st[j];
    }
  }
}

template <int R>
static int delta_group_scan_launch(const DeltaGroupArgs& a, int n_seqs, int threads, size_t smem, cudaStream_t stream) {
  static size_t set = 48 * 1024;
  if (smem > set) {
    if (cudaFuncSetAttribute(delta_group_scan_kernel<R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return ALOFA_ERR_LAUNCH;
    set = smem;
  }
  // an ordinary launch: its few long-lived CTAs would otherwise settle beside what is left of the kernel before, several to an SM (375 us a call, or 647)
  launch_whole(delta_group_scan_kernel<R>, dim3(a.H, n_seqs, (a.P + a.PC - 1) / a.PC), threads, smem, stream, a);
  return launch_status();
}

// The grouped scan: arguments as for alofa_delta_scan, with the tokens' pair words in place of kq, g and beta.
ALOFA_API int alofa_delta_group_scan(float* y, const float* v, int ldv, int v_off, const float* kn, const float* qn, const float* pairs, float* state, long long slot_stride,
                                     const int* q_start, const int* state_slots, int n_tokens, int n_seqs, int H, int G, int N, int P, int spread, cudaStream_t stream) {
  if (n_seqs <= 0 || n_tokens <= 0) return ALOFA_OK;
  if (H <= 0 || G <= 0 || H % G || N <= 0 || N > 1024 || P <= 0 || (uintptr_t)pairs % 16) return ALOFA_ERR_ARGUMENT;
  const int R = N <= 256 ? 8 : (N <= 512 ? 16 : 32);
  int NS = 1;
  while (NS * R < N) NS *= 2;
  int PC = 256 / NS;  // value channels per block, one per group of NS threads
  while (PC > 4 && PC / 2 >= P) PC /= 2;
  while (PC > 4 && PC * NS > 32 && (long long)H * n_seqs * ((P + PC - 1) / PC) < spread) PC /= 2;
  while (PC * NS < 32) PC *= 2;
  if (PC < 4) PC = 4;
  const int threads = (PC * NS + 31) / 32 * 32;
  const bool vec = N % 4 == 0 && P % 4 == 0 && PC % 4 == 0 && ldv % 4 == 0 && v_off % 4 == 0 && ((uintptr_t)v % 16 == 0) && ((uintptr_t)kn % 16 == 0) && ((uintptr_t)qn % 16 == 0);
  int TC = 16;
  while (TC > GROUP && (size_t)2 * TC * (2 * NS * R + PC + PAIR_WORDS) * sizeof(float) > 160 * 1024) TC /= 2;
  const size_t smem = (size_t)2 * TC * (2 * NS * R + PC + PAIR_WORDS) * sizeof(float);
  if (smem > 200 * 1024) return ALOFA_ERR_ARGUMENT;
  DeltaGroupArgs a = {y, v, ldv, v_off, kn, qn, pairs, state, slot_stride, q_start, state_slots, H, G, N, P, NS, PC, TC, vec ? 1 : 0};
  if (R == 8) return delta_group_scan_launch<8>(a, n_seqs, threads, smem, stream);
  if (R == 16) return delta_group_scan_launch<16>(a, n_seqs, threads, smem, stream);
  return delta_group_scan_launch<32>(a, n_seqs, threads, smem, stream);
}
