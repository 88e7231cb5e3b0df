// Linear attention with a matrix state per head: one decay number per head and token, an optional delta rule, an
// optional short convolution before it.  For a flat batch of portions, with H heads of key size d and value size dv over
// G query/key heads (head h reads query/key head h / (H / G)):
//
//   prep     from the projections' float32 sums u [T, ld]:
//              ``taps`` > 0: every channel of q, k, v passes a causal convolution over time (the last taps - 1 inputs
//              before a portion are the request's kept inputs in its state row) and then silu
//              ``unit``: every head of q and k divided by sqrt(sum(head^2) + unit_eps)
//              the first ``rotary_dim`` elements of every head of q and k turn by the token's position
//              q *= q_scale, k *= k_scale;  q, k are written with rows padded by zeros to DP elements a head
//              beta[t, h] = sigmoid(u_b);   g[t, h] = exp(-exp(A_log_h) softplus(u_a + dt_bias_h))
//   scan     per (request, head), token by token:
//              S <- g S;   x = v, or with the delta rule x = beta (v - S^T k);   S <- S + k x^T;   o = S^T q
//            S lives in the request's state row as [H, dv, d] (a value column's d elements side by side), float32, read
//            and written once per step
//   finish   out[t, h] = o / sqrt(mean(o^2) + eps) (* norm [dv]) * silu(gate) * out_scale, rounded once
//   step     scan and finish of single tokens, one per request, in one launch: a CTA owns a whole head
//
// Everything is float32 until ``finish``'s store.  The recurrence runs in the order of the tokens with a fixed order of
// additions, so a portion at once and token by token agree up to how the compiler contracts the same expressions.
#include "common.cuh"
#include "short_conv.cuh"
#include <math.h>

__device__ __forceinline__ void ls_st(void* p, int code, size_t i, float v) {
  if (code == QD_F32) reinterpret_cast<float*>(p)[i] = v;
  else reinterpret_cast<bf16*>(p)[i] = __float2bfloat16_rn(v);
}
__device__ __forceinline__ float ls_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ls_softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

// ------------------------------------------------------------------------------------------------------------ prep
#define LP_THREADS 128
#define LP_VCH 128            // channels of v a CTA takes
#define LP_MAX_TOKENS 8

struct LinearPrep {
  const float* u; long long ld;
  int T, H, G, d, dv, DP;
  int taps; const float* conv_w; float* state; long long state_stride, conv_off; int advance;
  const int *token_req, *cu_tokens, *slots;
  int unit; float unit_eps;
  int rotary_dim, pairing; const float *cos_t, *sin_t; const int* positions;
  float q_scale, k_scale;
  int b_off, a_off; const float *A_log, *dt_bias;             // columns of u, -1: not there
  float *q, *k, *v, *beta, *g;                                 // [T, G, DP] twice, [T, H * dv], [T, H] twice
  int v_slots, tokens;
};

// grid (2 G + v_slots + (gates ? 1 : 0), ceil(T / tokens)): a CTA takes ``tokens`` tokens of one query or key head, of
// LP_VCH channels of v, or of the gates.
__global__ void __launch_bounds__(LP_THREADS)
linear_prep_kernel(LinearPrep a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float lp_sm[];                    // [tokens][d], then [tokens] factors
  const int slot = blockIdx.x, t0 = blockIdx.y * a.tokens, nt = min(a.tokens, a.T - t0);
  const int tid = threadIdx.x;
  const int nq = a.G * a.d, C = 2 * nq + a.H * a.dv;
  auto channel = [&](int t, int c) {                  // what channel c of the stacked q | k | v is after conv and silu
    if (a.taps <= 0) return a.u[(size_t)t * a.ld + c];
    const int r = a.token_req[t];
    float* kept = a.taps > 1 ? a.state + (size_t)a.slots[r] * a.state_stride + a.conv_off : nullptr;
    const float y = short_conv_at(a.u, a.ld, C, a.taps, a.conv_w, kept, a.cu_tokens[r], t, c);
    // every request brings one token: this thread alone reads and writes channel c of its request's kept inputs
    if (a.advance) short_conv_advance(a.u, a.ld, C, a.taps, kept, t, t + 1, c);
    return ls_silu(y);
  };
  if (slot >= 2 * a.G + a.v_slots) {                  // the gates
    for (int e = tid; e < nt * a.H; e += LP_THREADS) {
      const int t = t0 + e / a.H, h = e - e / a.H * a.H;
      if (a.b_off >= 0) a.beta[(size_t)t * a.H + h] = 1.0f / (1.0f + expf(-a.u[(size_t)t * a.ld + a.b_off + h]));
      if (a.a_off >= 0)
        a.g[(size_t)t * a.H + h] = expf(-expf(a.A_log[h]) * ls_softplus(a.u[(size_t)t * a.ld + a.a_off + h] + a.dt_bias[h]));
    }
    return;
  }
  if (slot >= 2 * a.G) {                              // channels of v
    const int c0 = (slot - 2 * a.G) * LP_VCH, n = min(LP_VCH, a.H * a.dv - c0);
    for (int e = tid; e < nt * LP_VCH; e += LP_THREADS) {
      const int tt = e / LP_VCH, c = e - tt * LP_VCH;
      if (c < n) a.v[(size_t)(t0 + tt) * a.H * a.dv + c0 + c] = channel(t0 + tt, 2 * nq + c0 + c);
    }
    return;
  }
  const bool is_q = slot < a.G;
  const int head = is_q ? slot : slot - a.G, base = (is_q ? 0 : nq) + head * a.d, d = a.d;
  float* f = lp_sm + (size_t)a.tokens * d;
  for (int e = tid; e < nt * d; e += LP_THREADS) {
    const int tt = e / d;
    lp_sm[e] = channel(t0 + tt, base + e - tt * d);
  }
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31;
  for (int tt = warp; tt < nt; tt += LP_THREADS / 32) {
    float c = is_q ? a.q_scale : a.k_scale;
    if (a.unit) {
      float ss = 0.f;
      for (int i = lane; i < d; i += 32) ss = fmaf(lp_sm[tt * d + i], lp_sm[tt * d + i], ss);
      c *= 1.0f / sqrtf(warp_sum(ss) + a.unit_eps);
    }
    if (lane == 0) f[tt] = c;
  }
  __syncthreads();
  float* dst = is_q ? a.q : a.k;
  const int half = a.rotary_dim / 2;
  for (int e = tid; e < nt * a.DP; e += LP_THREADS) {
    const int tt = e / a.DP, i = e - tt * a.DP, t = t0 + tt;
    float y = 0.f;
    if (i < d) {
      const float* row = lp_sm + tt * d;
      y = row[i];
      if (i < 2 * half) {
        // the pair's first element turns to u cos - v sin, its second to v cos + u sin
        const int j = a.pairing == 1 ? (i < half ? i : i - half) : i >> 1;
        const bool first = a.pairing == 1 ? i < half : !(i & 1);
        const float other = row[a.pairing == 1 ? (first ? i + half : i - half) : i ^ 1];
        const size_t at = (size_t)a.positions[t] * half + j;
        y = first ? y * a.cos_t[at] - other * a.sin_t[at] : y * a.cos_t[at] + other * a.sin_t[at];
      }
      y *= f[tt];
    }
    dst[((size_t)t * a.G + head) * a.DP + i] = y;
  }
}

// grid (ceil(C / 256), requests): one thread per (request, channel) moves the channel's taps - 1 kept inputs on.
__global__ void __launch_bounds__(256)
linear_prep_state_kernel(const float* __restrict__ u, long long ld, int C, int taps, float* __restrict__ state,
                         long long state_stride, long long conv_off, const int* __restrict__ cu_tokens,
                         const int* __restrict__ slots) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, r = blockIdx.y;
  if (c >= C) return;
  short_conv_advance(u, ld, C, taps, state + (size_t)slots[r] * state_stride + conv_off, cu_tokens[r], cu_tokens[r + 1], c);
}

// u float32 [T, ld], a row = [q (G*d) | k (G*d) | v (H*dv) | ...]; conv_w float32 [2*G*d + H*dv, taps] (taps 0: no
// convolution, no silu, and v is not written); state rows ``state_stride`` apart with the (taps - 1) x C kept inputs at
// ``conv_off``, moved on by the portions when ``update_state``; b_off / a_off: columns of u of the step size's and the
// decay's logits (-1: none).
extern "C" int qd_linear_prep(const float* u, long long ld, int T, int n_requests, int H, int G, int d, int dv, int DP,
                              int taps, const float* conv_w, float* state, long long state_stride, long long conv_off,
                              const int* token_req, const int* cu_tokens, const int* slots, int update_state, int unit,
                              float unit_eps, int rotary_dim, int pairing, const float* cos_t, const float* sin_t,
                              const int* positions, float q_scale, float k_scale, int b_off, int a_off,
                              const float* A_log, const float* dt_bias, float* q, float* k, float* v, float* beta,
                              float* g, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0 || DP < d || DP > 256 || taps < 0 || (taps > 0 && (!conv_w || !v)) ||
      (taps > 1 && !state) || rotary_dim < 0 || rotary_dim > d || (rotary_dim & 1) ||
      (rotary_dim > 0 && (!cos_t || !sin_t || !positions)) || (b_off >= 0 && !beta) ||
      (a_off >= 0 && (!g || !A_log || !dt_bias)) || !q || !k || n_requests > 65535)
    return QD_ERR_UNSUPPORTED;
  const int tokens = T <= 32 ? 1 : T <= 128 ? 2 : LP_MAX_TOKENS;
  const int v_slots = taps > 0 ? (H * dv + LP_VCH - 1) / LP_VCH : 0;
  const int slots_x = 2 * G + v_slots + (b_off >= 0 || a_off >= 0 ? 1 : 0);
  if ((T + tokens - 1) / tokens > 65535) return QD_ERR_UNSUPPORTED;
  const int advance = update_state && taps > 1 && T == n_requests;       // single tokens, one per request
  const LinearPrep a = {u, ld, T, H, G, d, dv, DP, taps, conv_w, state, state_stride, conv_off, advance, token_req, cu_tokens,
                        slots, unit, unit_eps, rotary_dim, pairing, cos_t, sin_t, positions, q_scale, k_scale, b_off, a_off,
                        A_log, dt_bias, q, k, v, beta, g, v_slots, tokens};
  const size_t smem = ((size_t)tokens * d + tokens) * sizeof(float);      // at most 8 * 257 floats
  qd_launch(linear_prep_kernel, dim3(slots_x, (T + tokens - 1) / tokens), dim3(LP_THREADS), smem, stream, a);
  if (update_state && taps > 1 && !advance) {
    const int C = 2 * G * d + H * dv;
    qd_launch(linear_prep_state_kernel, dim3((C + 255) / 256, n_requests), dim3(256), 0, stream, u, ld, C, taps, state,
              state_stride, conv_off, cu_tokens, slots);
  }
  return qd_last_error();
}

// ------------------------------------------------------------------------------------------------------------ scan
// Thread (x = tid & 3, column = tid >> 2) keeps the elements i = 16 m + 4 x + c (c < 4, m < NI / 4) of one value
// column of S in registers; the four threads of a column are neighbouring lanes.
#define LS_GROUP 16           // tokens of operands in shared memory at a time (two such groups in flight)
#define LS_COLS 32            // value columns a CTA owns
#define LS_THREADS (4 * LS_COLS)

struct LinearScan {
  const float *q, *k;                     // [T, G, DP]
  const float* v; long long ldv;          // row t at t * ldv, head h at + h * dv
  const float* g; int g_ld;               // [T, H] (g_ld = H), or one number per head (g_ld = 0)
  const float* beta;                      // [T, H] (delta rule)
  int H, G, d, dv;
  float* state; long long state_stride, s_off; int vec;         // vec: rows of d elements start on 16-byte boundaries
  const int *cu_tokens, *slots;
  int write_state;
};

template <int NI>
__device__ __forceinline__ void ls_load_state(float (&s)[NI], const float* col, int x, int d, bool live, bool vec) {
#pragma unroll
  for (int m = 0; m < NI / 4; m++) {
    const int i = 16 * m + 4 * x;
    if (vec) {
      const float4 t = live && i < d ? *reinterpret_cast<const float4*>(col + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[4 * m] = t.x; s[4 * m + 1] = t.y; s[4 * m + 2] = t.z; s[4 * m + 3] = t.w;
    } else {
#pragma unroll
      for (int c = 0; c < 4; c++) s[4 * m + c] = live && i + c < d ? col[i + c] : 0.f;
    }
  }
}
template <int NI>
__device__ __forceinline__ void ls_store_state(const float (&s)[NI], float* col, int x, int d, bool vec) {
#pragma unroll
  for (int m = 0; m < NI / 4; m++) {
    const int i = 16 * m + 4 * x;
    if (vec) {
      if (i < d) *reinterpret_cast<float4*>(col + i) = make_float4(s[4 * m], s[4 * m + 1], s[4 * m + 2], s[4 * m + 3]);
    } else {
#pragma unroll
      for (int c = 0; c < 4; c++)
        if (i + c < d) col[i + c] = s[4 * m + c];
    }
  }
}

// One token: the state moves on, and this thread's share of S^T q comes back.  kr / qr: the token's k and q (DP elements,
// 16-byte aligned).
template <int NI, bool DELTA>
__device__ __forceinline__ float ls_token(float (&s)[NI], const float* kr, const float* qr, float v, float g, float beta, int x) {
  float4 kk[NI / 4];
#pragma unroll
  for (int m = 0; m < NI / 4; m++) kk[m] = *reinterpret_cast<const float4*>(kr + 16 * m + 4 * x);
  float w = v;
  if (DELTA) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int m = 0; m < NI / 4; m++) {
      a.x = fmaf(s[4 * m], kk[m].x, a.x);
      a.y = fmaf(s[4 * m + 1], kk[m].y, a.y);
      a.z = fmaf(s[4 * m + 2], kk[m].z, a.z);
      a.w = fmaf(s[4 * m + 3], kk[m].w, a.w);
    }
    float dot = (a.x + a.y) + (a.z + a.w);
    dot += __shfl_xor_sync(0xffffffffu, dot, 2);
    dot += __shfl_xor_sync(0xffffffffu, dot, 1);
    w = beta * fmaf(-g, dot, v);                      // (g S)^T k = g (S^T k)
  }
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int m = 0; m < NI / 4; m++) {
    const float4 qq = *reinterpret_cast<const float4*>(qr + 16 * m + 4 * x);
    s[4 * m] = fmaf(kk[m].x, w, g * s[4 * m]);
    s[4 * m + 1] = fmaf(kk[m].y, w, g * s[4 * m + 1]);
    s[4 * m + 2] = fmaf(kk[m].z, w, g * s[4 * m + 2]);
    s[4 * m + 3] = fmaf(kk[m].w, w, g * s[4 * m + 3]);
    o.x = fmaf(s[4 * m], qq.x, o.x);
    o.y = fmaf(s[4 * m + 1], qq.y, o.y);
    o.z = fmaf(s[4 * m + 2], qq.z, o.z);
    o.w = fmaf(s[4 * m + 3], qq.w, o.w);
  }
  return (o.x + o.y) + (o.z + o.w);
}

__device__ __forceinline__ void ls_cp16(float* smem, const float* gmem, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem),
               "r"(there ? 16 : 0));
}
__device__ __forceinline__ void ls_cp4(float* smem, const float* gmem, bool there) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem),
               "r"(there ? 4 : 0));
}

// grid (ceil(dv / LS_COLS), H, requests).  out float32 [T, H * dv] dense.
template <int NI, bool DELTA>
__global__ void __launch_bounds__(LS_THREADS)
linear_scan_kernel(LinearScan a, float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DP = 4 * NI, STAGE = LS_GROUP * (2 * DP + LS_COLS + 2);
  extern __shared__ __align__(16) float ls_sm[];      // two stages of [q][k][v][g][beta]
  const int tid = threadIdx.x, x = tid & 3, jl = tid >> 2;
  const int h = blockIdx.y, req = blockIdx.z, j0 = blockIdx.x * LS_COLS, j = j0 + jl;
  const int gk = h / (a.H / a.G), d = a.d, dv = a.dv;
  const bool live = j < dv;
  const int t0 = a.cu_tokens[req], t1 = a.cu_tokens[req + 1];
  if (t0 >= t1) return;
  float* col = a.state + (size_t)a.slots[req] * a.state_stride + a.s_off + ((size_t)h * dv + (live ? j : 0)) * d;
  float s[NI];
  // Operands of the tokens tb .. tb + LS_GROUP - 1; places past the portion's end hold q = k = v = beta = 0 and g = 1,
  // which leave the state as it is.
  auto fetch = [&](int tb, int stage) {
    float* qs = ls_sm + stage * STAGE;
    float* ks = qs + LS_GROUP * DP;
    float* vs = ks + LS_GROUP * DP;
    float* gs = vs + LS_GROUP * LS_COLS;
    float* bs = gs + LS_GROUP;
    for (int e = tid; e < LS_GROUP * NI; e += LS_THREADS) {
      const int tt = e / NI, c = (e - tt * NI) * 4;
      const bool there = tb + tt < t1;
      const size_t src = there ? ((size_t)(tb + tt) * a.G + gk) * DP + c : 0;
      ls_cp16(qs + tt * DP + c, a.q + src, there);
      ls_cp16(ks + tt * DP + c, a.k + src, there);
    }
    for (int e = tid; e < LS_GROUP * LS_COLS; e += LS_THREADS) {
      const int tt = e / LS_COLS, c = e - tt * LS_COLS;
      const bool there = tb + tt < t1 && j0 + c < dv;
      ls_cp4(vs + e, there ? a.v + (size_t)(tb + tt) * a.ldv + (size_t)h * dv + j0 + c : a.v, there);
    }
    if (tid < LS_GROUP) {
      const bool there = tb + tid < t1;
      if (there) ls_cp4(gs + tid, a.g + (a.g_ld ? (size_t)(tb + tid) * a.g_ld : 0) + h, true);
      else gs[tid] = 1.0f;
      if (DELTA) ls_cp4(bs + tid, there ? a.beta + (size_t)(tb + tid) * a.H + h : a.beta, there);
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  fetch(t0, 0);
  ls_load_state<NI>(s, col, x, d, live, a.vec);
  int stage = 0;
  for (int tb = t0; tb < t1; tb += LS_GROUP, stage ^= 1) {
    if (tb + LS_GROUP < t1) {
      fetch(tb + LS_GROUP, stage ^ 1);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    const float* qs = ls_sm + stage * STAGE;
    const float* ks = qs + LS_GROUP * DP;
    const float* vs = ks + LS_GROUP * DP;
    const float* gs = vs + LS_GROUP * LS_COLS;
    const float* bs = gs + LS_GROUP;
    const int nt = min(LS_GROUP, t1 - tb);
    for (int q4 = 0; q4 < nt; q4 += 4) {
      float acc[4];
#pragma unroll
      for (int p = 0; p < 4; p++) {
        const int tt = q4 + p;
        acc[p] = ls_token<NI, DELTA>(s, ks + tt * DP, qs + tt * DP, vs[tt * LS_COLS + jl], gs[tt], DELTA ? bs[tt] : 0.f, x);
      }
      // The four threads of a column add up their shares of four tokens at once; thread x ends with token q4 + x's sum,
      // by the same tree of additions for every place of a token.
      const bool hi2 = x & 2, hi1 = x & 1;
      const float r0 = (hi2 ? acc[2] : acc[0]) + __shfl_xor_sync(0xffffffffu, hi2 ? acc[0] : acc[2], 2);
      const float r1 = (hi2 ? acc[3] : acc[1]) + __shfl_xor_sync(0xffffffffu, hi2 ? acc[1] : acc[3], 2);
      const float o = (hi1 ? r1 : r0) + __shfl_xor_sync(0xffffffffu, hi1 ? r0 : r1, 1);
      if (q4 + x < nt && live) out[(size_t)(tb + q4 + x) * a.H * dv + (size_t)h * dv + j] = o;
    }
    __syncthreads();                                  // this stage is overwritten by the next turn's fetch
  }
  if (a.write_state && live) ls_store_state<NI>(s, col, x, d, a.vec);
}

// ---------------------------------------------------------------------------------------------------------- finish
struct LinearFinish {
  const float* gate; long long gate_ld;   // float32 logits, head h's at + h * dv; silu is taken here
  const float* norm;                      // [dv] or null
  float eps, out_scale;
  void* out; int out_dtype; long long out_stride;
};

// grid (ceil(T * H / 8)), a warp per (token, head).
__global__ void __launch_bounds__(256)
linear_finish_kernel(const float* __restrict__ o, int T, int H, int dv, LinearFinish f) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= (long long)T * H) return;
  const int t = (int)(item / H), h = (int)(item - (long long)t * H);
  const float* row = o + (size_t)item * dv;
  float ss = 0.f;
  for (int i = lane; i < dv; i += 32) { const float y = row[i]; ss = fmaf(y, y, ss); }
  const float c = f.out_scale / sqrtf(warp_sum(ss) / (float)dv + f.eps);
  const float* gate = f.gate + (size_t)t * f.gate_ld + (size_t)h * dv;
  for (int i = lane; i < dv; i += 32)
    ls_st(f.out, f.out_dtype, (size_t)t * f.out_stride + (size_t)h * dv + i,
          row[i] * c * (f.norm ? f.norm[i] : 1.0f) * ls_silu(gate[i]));
}

// ------------------------------------------------------------------------------------------------------------ step
// grid (H, requests), 4 * (columns at a time) threads, at most 512.  Request r's token is token r.
#define LS_STEP_THREADS 512

template <int NI, bool DELTA>
__global__ void __launch_bounds__(LS_STEP_THREADS)
linear_step_kernel(LinearScan a, LinearFinish f) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DP = 4 * NI;
  extern __shared__ float st_sm[];                    // [dv] outputs, then 40 of scratch
  const int tid = threadIdx.x, x = tid & 3, jl = tid >> 2, cols = blockDim.x >> 2;
  const int h = blockIdx.x, t = blockIdx.y, d = a.d, dv = a.dv, gk = h / (a.H / a.G);
  float* S = a.state + (size_t)a.slots[t] * a.state_stride + a.s_off + (size_t)h * dv * d;
  const float* kr = a.k + ((size_t)t * a.G + gk) * DP;
  const float* qr = a.q + ((size_t)t * a.G + gk) * DP;
  const float g = a.g[(a.g_ld ? (size_t)t * a.g_ld : 0) + h];
  const float beta = DELTA ? a.beta[(size_t)t * a.H + h] : 0.f;
  float ss = 0.f;
  for (int j0 = 0; j0 < dv; j0 += cols) {             // every thread takes every turn: the shuffles need them all
    const int j = j0 + jl;
    const bool live = j < dv;
    float* col = S + (size_t)(live ? j : 0) * d;
    float s[NI];
    ls_load_state<NI>(s, col, x, d, live, a.vec);
    const float v = live ? a.v[(size_t)t * a.ldv + (size_t)h * dv + j] : 0.f;
    float o = ls_token<NI, DELTA>(s, kr, qr, v, g, beta, x);
    o += __shfl_xor_sync(0xffffffffu, o, 2);
    o += __shfl_xor_sync(0xffffffffu, o, 1);
    if (live && x == 0) {
      st_sm[j] = o;
      ss = fmaf(o, o, ss);
    }
    if (a.write_state && live) ls_store_state<NI>(s, col, x, d, a.vec);
  }
  const float c = f.out_scale / sqrtf(block_sum(ss, st_sm + dv) / (float)dv + f.eps);     // meets the writes of st_sm, too
  const float* gate = f.gate + (size_t)t * f.gate_ld + (size_t)h * dv;
  for (int i = tid; i < dv; i += blockDim.x)
    ls_st(f.out, f.out_dtype, (size_t)t * f.out_stride + (size_t)h * dv + i,
          st_sm[i] * c * (f.norm ? f.norm[i] : 1.0f) * ls_silu(gate[i]));
}

// ------------------------------------------------------------------------------------------------------- launchers
// q, k float32 [T, G, DP], DP the padded head size: the smallest of 16, 32, 48, 64, 96, 128, 256 that holds d; v rows
// ``ldv`` apart; g float32 [T, H] (g_ld = H) or [H] (g_ld = 0); beta float32 [T, H]: the delta rule, or null;
// state float32 rows ``state_stride`` apart, the heads' matrices [H, dv, d] at ``s_off``; o_buf float32 [T, H * dv]
// (unused when every request brings one token); gate float32 rows ``gate_ld`` apart; norm float32 [dv] or null.
extern "C" int qd_linear_scan(const float* q, const float* k, const float* v, long long ldv, const float* g, int g_ld,
                              const float* beta, int T, int n_requests, int H, int G, int d, int dv, int DP,
                              float* state, long long state_stride, long long s_off, const int* cu_tokens,
                              const int* slots, int write_state, float* o_buf, const float* gate, long long gate_ld,
                              const float* norm, float eps, float out_scale, void* out, int out_dtype,
                              long long out_stride, cudaStream_t stream) {
  if (T <= 0 || n_requests <= 0) return 0;
  if (H <= 0 || H > 65535 || n_requests > 65535 || G <= 0 || H % G || d <= 0 || dv <= 0 || dv > 8192 || d > DP ||
      !state || !gate || (g_ld && g_ld != H) || (out_dtype != QD_F32 && out_dtype != QD_BF16))
    return QD_ERR_UNSUPPORTED;
  const bool single = T == n_requests;                // every request has at least one token
  if (!single && !o_buf) return QD_ERR_UNSUPPORTED;
  if (((uintptr_t)q | (uintptr_t)k) & 15) return QD_ERR_UNSUPPORTED;
  const int vec = d % 4 == 0 && state_stride % 4 == 0 && s_off % 4 == 0 && !((uintptr_t)state & 15);
  const LinearScan a = {q, k, v, ldv, g, g_ld, beta, H, G, d, dv, state, state_stride, s_off, vec, cu_tokens, slots, write_state};
  const LinearFinish f = {gate, gate_ld, norm, eps, out_scale, out, out_dtype, out_stride};
  const int cols = (dv + 7) / 8 * 8 < LS_STEP_THREADS / 4 ? (dv + 7) / 8 * 8 : LS_STEP_THREADS / 4;
  const size_t step_smem = ((size_t)dv + 40) * sizeof(float);
#define LS_GO2(NI, DELTA)                                                                                             \
  do {                                                                                                                \
    if (single) {                                                                                                     \
      qd_launch(linear_step_kernel<NI, DELTA>, dim3(H, n_requests), dim3(4 * cols), step_smem, stream, a, f);         \
    } else {                                                                                                          \
      const size_t smem = (size_t)2 * LS_GROUP * (8 * NI + LS_COLS + 2) * sizeof(float);                              \
      static bool raised = false;                                                                                     \
      if (!raised && smem > 48 * 1024) {                                                                              \
        cudaFuncSetAttribute(linear_scan_kernel<NI, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
        raised = true;                                                                                                \
      }                                                                                                               \
      qd_launch(linear_scan_kernel<NI, DELTA>, dim3((dv + LS_COLS - 1) / LS_COLS, H, n_requests), dim3(LS_THREADS), smem, \
                stream, a, o_buf);                                                                                    \
    }                                                                                                                 \
  } while (0)
#define LS_GO(NI) do { if (beta) LS_GO2(NI, true); else LS_GO2(NI, false); } while (0)
  switch (DP) {
    case 16: LS_GO(4); break;
    case 32: LS_GO(8); break;
    case 48: LS_GO(12); break;
    case 64: LS_GO(16); break;
    case 96: LS_GO(24); break;
    case 128: LS_GO(32); break;
    case 256: LS_GO(64); break;
    default: return QD_ERR_UNSUPPORTED;
  }
#undef LS_GO
#undef LS_GO2
  if (!single)
    qd_launch(linear_finish_kernel, dim3((unsigned)(((long long)T * H + 7) / 8)), dim3(256), 0, stream, (const float*)o_buf,
              T, H, dv, f);
  return qd_last_error();
}
