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
//   finish   out[t, h] = o / sqrt(mean(o^2) + eps) (* norm) * silu(gate) (or sigmoid) * out_scale, rounded once
//   step     scan and finish of single tokens, one per request, in one launch: a CTA owns a whole head
//
// With exponential gates (``ExpGates``) a head has a log input gate i = cap tanh((u_i + ib) / cap), a log forget gate
// f = logsigmoid(cap tanh((u_f + fb) / cap)) and a running maximum m (0 for a fresh request), m' = max(f + m, i):
//   S <- e^(f + m - m') S + e^(i - m') k v^T,   n <- e^(f + m - m') n + e^(i - m') k,
//   o = S^T q / (max(|n . q|, e^-m') + 1e-6)
// n is one more column of S whose value is always 1 (the state then is [H, dv + 1, d], and m is kept beside it);
// ``gates`` makes the decays, e^(i - m') and e^-m' of portions, ``prep`` multiplies k by e^(i - m'), ``finish`` divides.
// A step of single tokens does all of it in its one launch.
//
// Everything is float32 until ``finish``'s store.  The order of every sum depends on the sizes and on a token's place in its
// portion only: however a prompt is cut, the results agree up to the rounding of float32 sums.
#include "common.cuh"
#include "short_conv.cuh"
#include <math.h>

__device__ __forceinline__ void ls_st(void* p, int code, size_t i, float v) {
  if (code == QD_F32) reinterpret_cast<float*>(p)[i] = v;
  else reinterpret_cast<bf16*>(p)[i] = __float2bfloat16_rn(v);
}
__device__ __forceinline__ float ls_silu(float z) { return z / (1.0f + expf(-z)); }
// What the output gate multiplies by: silu (0) or sigmoid (1) of the logit.
__device__ __forceinline__ float ls_gate(float z, int kind) { return (kind ? 1.0f : z) / (1.0f + expf(-z)); }
__device__ __forceinline__ float ls_softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

// ------------------------------------------------------------------------------------------------------------ prep
#define LP_THREADS 128
#define LP_VCH 128            // channels of v a CTA takes
#define LP_MAX_TOKENS 16

struct LinearPrep {
  const float* u; long long ld;
  int T, H, G, d, dv, DP;
  int taps; const float* conv_w; float* state; long long state_stride, conv_off; int advance;
  const int *token_req, *cu_tokens, *slots;
  int unit; float unit_eps;
  int rotary_dim, pairing; const float *cos_t, *sin_t; const int* positions;
  float q_scale, k_scale;
  int b_off, a_off; const float *A_log, *dt_bias;             // columns of u, -1: not there
  const float* k_mul;                                          // [T, G]: one more factor of k, or null
  float *q, *k, *v, *beta, *g;                                 // [T, G, DP] twice, [T, H * dv], [T, H] twice
  int v_slots, tokens;
};

// grid (2 G + v_slots + (gates ? 1 : 0), ceil(T / tokens)): a CTA takes ``tokens`` tokens of one query or key head, of
// LP_VCH channels of v, or of the gates.
__global__ void __launch_bounds__(LP_THREADS)
linear_prep_kernel(LinearPrep a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float lp_sm[];                    // [tokens][d] outputs, [tokens] factors, then the inputs' rows
  const int slot = blockIdx.x, t0 = blockIdx.y * a.tokens, nt = min(a.tokens, a.T - t0);
  const int tid = threadIdx.x;
  const int nq = a.G * a.d, C = 2 * nq + a.H * a.dv;
  const int back = a.taps > 1 ? a.taps - 1 : 0, first = max(0, t0 - back);     // the rows of u this CTA's tokens read
  float* rows = lp_sm + (size_t)a.tokens * a.d + a.tokens;
  // Columns c0 .. c0 + n - 1 of those rows into shared memory, ``w`` apart.
  auto fetch = [&](int c0, int n, int w) {
    for (int e = tid; e < (t0 + nt - first) * w; e += LP_THREADS) {
      const int rr = e / w, c = e - rr * w;
      if (c < n) rows[e] = a.u[(size_t)(first + rr) * a.ld + c0 + c];
    }
    __syncthreads();
  };
  // What channel c0 + c of the stacked q | k | v is after convolution and silu, from the fetched rows.
  auto channel = [&](int t, int c0, int c, int w) {
    if (a.taps <= 0) return rows[(t - first) * w + c];
    const int r = a.token_req[t], begin = a.cu_tokens[r], li = t - begin, ch = c0 + c;
    float* kept = a.taps > 1 ? a.state + (size_t)a.slots[r] * a.state_stride + a.conv_off : nullptr;
    float y = 0.f;
    for (int j = 0; j < a.taps; j++) {
      const int s = li - (a.taps - 1) + j;            // the tap's place in the portion; before it: a kept input
      const float v = s >= 0 ? rows[(begin + s - first) * w + c] : kept[(size_t)(a.taps - 1 + s) * C + ch];
      y = fmaf(a.conv_w[(size_t)ch * a.taps + j], v, y);
    }
    // every request brings one token: this thread alone reads and writes the channel's kept inputs of its request
    if (a.advance) short_conv_advance(a.u, a.ld, C, a.taps, kept, t, t + 1, ch);
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
    fetch(2 * nq + c0, n, LP_VCH);
    for (int e = tid; e < nt * LP_VCH; e += LP_THREADS) {
      const int tt = e / LP_VCH, c = e - tt * LP_VCH;
      if (c < n) a.v[(size_t)(t0 + tt) * a.H * a.dv + c0 + c] = channel(t0 + tt, 2 * nq + c0, c, LP_VCH);
    }
    return;
  }
  const bool is_q = slot < a.G;
  const int head = is_q ? slot : slot - a.G, base = (is_q ? 0 : nq) + head * a.d, d = a.d;
  float* f = lp_sm + (size_t)a.tokens * d;
  fetch(base, d, d);
  for (int e = tid; e < nt * d; e += LP_THREADS) {
    const int tt = e / d;
    lp_sm[e] = channel(t0 + tt, base, e - tt * d, d);
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
    if (!is_q && a.k_mul) c *= a.k_mul[(size_t)(t0 + tt) * a.G + head];
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
// decay's logits (-1: none); k_mul float32 [T, G] (null: none): multiplies k's heads.
extern "C" int qd_linear_prep(const float* u, long long ld, int T, int n_requests, int H, int G, int d, int dv, int DP,
                              int taps, const float* conv_w, float* state, long long state_stride, long long conv_off,
                              const int* token_req, const int* cu_tokens, const int* slots, int update_state, int unit,
                              float unit_eps, int rotary_dim, int pairing, const float* cos_t, const float* sin_t,
                              const int* positions, float q_scale, float k_scale, int b_off, int a_off,
                              const float* A_log, const float* dt_bias, const float* k_mul, float* q, float* k, float* v,
                              float* beta, float* g, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || dv <= 0 || DP < d || DP > 256 || taps < 0 || (taps > 0 && (!conv_w || !v)) ||
      (taps > 1 && !state) || rotary_dim < 0 || rotary_dim > d || (rotary_dim & 1) ||
      (rotary_dim > 0 && (!cos_t || !sin_t || !positions)) || (b_off >= 0 && !beta) ||
      (a_off >= 0 && (!g || !A_log || !dt_bias)) || !q || !k || n_requests > 65535)
    return QD_ERR_UNSUPPORTED;
  int tokens = T <= 32 ? 1 : T <= 128 ? 2 : LP_MAX_TOKENS;
  const int v_slots = taps > 0 ? (H * dv + LP_VCH - 1) / LP_VCH : 0;
  const int slots_x = 2 * G + v_slots + (b_off >= 0 || a_off >= 0 ? 1 : 0);
  const int width = v_slots && LP_VCH > d ? LP_VCH : d;
  auto bytes = [&](int n) { return ((size_t)n * d + n + (size_t)(n + (taps > 1 ? taps - 1 : 0)) * width) * sizeof(float); };
  while (tokens > 1 && bytes(tokens) > 48 * 1024) tokens /= 2;
  const size_t smem = bytes(tokens);
  if (smem > 200 * 1024 || (T + tokens - 1) / tokens > 65535) return QD_ERR_UNSUPPORTED;
  static size_t raised = 48 * 1024;
  if (smem > raised) {
    cudaFuncSetAttribute(linear_prep_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    raised = smem;
  }
  const int advance = update_state && taps > 1 && T == n_requests;       // single tokens, one per request
  const LinearPrep a = {u, ld, T, H, G, d, dv, DP, taps, conv_w, state, state_stride, conv_off, advance, token_req, cu_tokens,
                        slots, unit, unit_eps, rotary_dim, pairing, cos_t, sin_t, positions, q_scale, k_scale, b_off, a_off,
                        A_log, dt_bias, k_mul, q, k, v, beta, g, v_slots, tokens};
  qd_launch(linear_prep_kernel, dim3(slots_x, (T + tokens - 1) / tokens), dim3(LP_THREADS), smem, stream, a);
  if (update_state && taps > 1 && !advance) {
    const int C = 2 * G * d + H * dv;
    qd_launch(linear_prep_state_kernel, dim3((C + 255) / 256, n_requests), dim3(256), 0, stream, u, ld, C, taps, state,
              state_stride, conv_off, cu_tokens, slots);
  }
  return qd_last_error();
}

// ----------------------------------------------------------------------------------------------- exponential gates
#define LS_NRM_EPS 1e-6f      // beside the larger of |n . q| and e^-m in the denominator
struct ExpGates {
  const float* u; long long ld; int i_off, f_off;             // the logits: row t at t * ld, head h at i_off + h, f_off + h
  const float *ib, *fb; float cap;                            // [H] each
  long long m_off;                                            // head h's maximum is at m_off + h of a state row
  int on;
};
__device__ __forceinline__ void exp_gate_logs(const ExpGates& a, float ui, float uf, int h, float& i, float& f) {
  i = a.cap * tanhf((ui + a.ib[h]) / a.cap);
  const float z = a.cap * tanhf((uf + a.fb[h]) / a.cap);
  f = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// grid (H, requests): the maxima of a portion by a scan over (sum of f, maximum): what a run of tokens does to m is
// m -> max(F + m, M), and runs compose.  A thread takes one token of as many as the CTA has threads; warps scan their 32, then one another's.
// Every factor is made from the maxima as they are handed on, so what rounds in the scan cancels between a token and the next.
#define LG_TOKENS 1024
__global__ void __launch_bounds__(LG_TOKENS)
linear_exp_gates_kernel(ExpGates a, int H, float* __restrict__ state, long long state_stride,
                        const int* __restrict__ cu_tokens, const int* __restrict__ slots, int write_state,
                        float* __restrict__ g, float* __restrict__ in, float* __restrict__ low) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float wF[32], wM[32], ms[LG_TOKENS + 1];
  const int h = blockIdx.x, req = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = cu_tokens[req], t1 = cu_tokens[req + 1];
  if (t0 >= t1) return;
  float* kept = state + (size_t)slots[req] * state_stride + a.m_off + h;
  float m0 = *kept;
  float ui = 0.f, uf = 0.f;                           // the logits of the turn ahead are under way during this one
  auto fetch = [&](int t) {
    if (t < t1) { ui = a.u[(size_t)t * a.ld + a.i_off + h]; uf = a.u[(size_t)t * a.ld + a.f_off + h]; }
  };
  fetch(t0 + tid);
  const int at_once = blockDim.x, warps = at_once >> 5;
  for (int tb = t0; tb < t1; tb += at_once) {
    const int t = tb + tid;
    float i = -INFINITY, f = 0.f;                     // past the end: m stays as it is
    if (t < t1) exp_gate_logs(a, ui, uf, h, i, f);
    fetch(t + at_once);
    float F = f, M = i;                               // of the warp's tokens up to this one
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) {
        M = fmaxf(Mp + F, M);
        F += Fp;
      }
    }
    if (lane == 31) { wF[warp] = F; wM[warp] = M; }
    __syncthreads();
    // what the warps before this one make of m0: lane w holds warp w's run; neighbours compose, five times
    float Fw = lane < warp && lane < warps ? wF[lane] : 0.f, Mw = lane < warp && lane < warps ? wM[lane] : -INFINITY;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float Fr = __shfl_down_sync(0xffffffffu, Fw, o), Mr = __shfl_down_sync(0xffffffffu, Mw, o);
      Mw = fmaxf(Mw + Fr, Mr);
      Fw += Fr;
    }
    const float before = fmaxf(__shfl_sync(0xffffffffu, Fw, 0) + m0, __shfl_sync(0xffffffffu, Mw, 0));
    const float m = fmaxf(F + before, M);
    if (tid == 0) ms[0] = m0;
    ms[tid + 1] = m;
    __syncthreads();
    if (t < t1) {
      const size_t at = (size_t)t * H + h;
      g[at] = expf(f + (ms[tid] - m));
      in[at] = expf(i - m);
      low[at] = expf(-m);
    }
    m0 = ms[at_once];
  }
  if (write_state && tid == 0) *kept = m0;
}

// From the logits' columns of u: g = e^(f + m - m'), in = e^(i - m') and low = e^-m', float32 [T, H]; the maxima of the
// requests' state rows are moved on when ``write_state``.
extern "C" int qd_linear_exp_gates(const float* u, long long ld, int i_off, int f_off, const float* ib, const float* fb,
                                   float cap, int T, int n_requests, int H, float* state, long long state_stride,
                                   long long m_off, const int* cu_tokens, const int* slots, int write_state, float* g,
                                   float* in, float* low, cudaStream_t stream) {
  if (T <= 0 || n_requests <= 0) return 0;
  if (H <= 0 || n_requests > 65535 || !ib || !fb || !(cap > 0.f) || !state || !g || !in || !low) return QD_ERR_UNSUPPORTED;
  const ExpGates a = {u, ld, i_off, f_off, ib, fb, cap, m_off, 1};
  qd_launch(linear_exp_gates_kernel, dim3(H, n_requests), dim3(T < LG_TOKENS ? (T + 31) / 32 * 32 : LG_TOKENS), 0, stream, a, H, state, state_stride, cu_tokens, slots,
            write_state, g, in, low);
  return qd_last_error();
}

// ------------------------------------------------------------------------------------------------------------ scan
#define LS_GROUP 16           // tokens of operands in shared memory at a time (two such groups in flight)

struct LinearScan {
  const float *q, *k;                     // [T, G, DP]
  const float* v; long long ldv;          // row t at t * ldv, head h at + h * dv
  const float* g; int g_ld;               // [T, H] (g_ld = H), or one number per head (g_ld = 0)
  const float* beta;                      // [T, H] (delta rule)
  const float* coef;                      // [T, H, LS_COEF] (delta rule, portions)
  int H, G, d, dv;
  float* state; long long state_stride, s_off; int vec;         // vec: rows of d elements start on 16-byte boundaries
  const int *cu_tokens, *slots;
  int write_state;
  int nrm; float* nq;                     // nrm: one more column whose value is 1; its outputs [T, H]
  // single tokens: where q's and k's rows are, if they are not padded (``raw``), and what they are still multiplied by
  int raw; long long q_ld; float q_scale, k_scale;
};

// Two float32 numbers that one instruction works on (each rounded as by itself).
typedef unsigned long long f2;
__device__ __forceinline__ f2 f2_make(float lo, float hi) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float f2_lo(f2 v) { return __uint_as_float((unsigned)v); }
__device__ __forceinline__ float f2_hi(f2 v) { return __uint_as_float((unsigned)(v >> 32)); }
// PACKED: one instruction for both; else two (a loop that waits for latencies rather than for issue slots is better off).
template <bool PACKED>
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) {
  if (!PACKED) return f2_make(fmaf(f2_lo(a), f2_lo(b), f2_lo(c)), fmaf(f2_hi(a), f2_hi(b), f2_hi(c)));
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
template <bool PACKED>
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) {
  if (!PACKED) return f2_make(f2_lo(a) * f2_lo(b), f2_hi(a) * f2_hi(b));
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f2 f2_add(f2 a, f2 b) { return f2_make(f2_lo(a) + f2_lo(b), f2_hi(a) + f2_hi(b)); }

// A thread's share of one value column of S: lane x of X takes the E elements i = 4 X m + 4 x + c (c < 4, m < E / 4), two to a
// register pair.
template <int E, int X>
__device__ __forceinline__ void ls_load_state(f2 (&s)[E / 2], const float* col, int x, int d, bool live, bool vec) {
#pragma unroll
  for (int m = 0; m < E / 4; m++) {
    const int i = 4 * X * m + 4 * x;
    if (vec) {
      const ulonglong2 t = live && i < d ? *reinterpret_cast<const ulonglong2*>(col + i) : make_ulonglong2(0, 0);
      s[2 * m] = t.x;
      s[2 * m + 1] = t.y;
    } else {
#pragma unroll
      for (int c = 0; c < 2; c++)
        s[2 * m + c] = f2_make(live && i + 2 * c < d ? col[i + 2 * c] : 0.f, live && i + 2 * c + 1 < d ? col[i + 2 * c + 1] : 0.f);
    }
  }
}
template <int E, int X>
__device__ __forceinline__ void ls_store_state(const f2 (&s)[E / 2], float* col, int x, int d, bool vec) {
#pragma unroll
  for (int m = 0; m < E / 4; m++) {
    const int i = 4 * X * m + 4 * x;
    if (vec) {
      if (i < d) *reinterpret_cast<ulonglong2*>(col + i) = make_ulonglong2(s[2 * m], s[2 * m + 1]);
    } else {
#pragma unroll
      for (int c = 0; c < 2; c++) {
        if (i + 2 * c < d) col[i + 2 * c] = f2_lo(s[2 * m + c]);
        if (i + 2 * c + 1 < d) col[i + 2 * c + 1] = f2_hi(s[2 * m + c]);
      }
    }
  }
}

// This thread's share of S^T k of a column: s . k over its elements.
template <int E, bool PACKED>
__device__ __forceinline__ float ls_dot(const f2 (&s)[E / 2], const f2 (&k)[E / 2]) {
  f2 a = f2_mul<PACKED>(s[0], k[0]), b = f2_mul<PACKED>(s[1], k[1]);
#pragma unroll
  for (int m = 1; m < E / 4; m++) {
    a = f2_fma<PACKED>(s[2 * m], k[2 * m], a);
    b = f2_fma<PACKED>(s[2 * m + 1], k[2 * m + 1], b);
  }
  a = f2_add(a, b);
  return f2_lo(a) + f2_hi(a);
}
// s <- g s + w k
template <int E, bool PACKED>
__device__ __forceinline__ void ls_move(f2 (&s)[E / 2], const f2 (&k)[E / 2], float w, float g) {
  const f2 ww = f2_make(w, w), gg = f2_make(g, g);
#pragma unroll
  for (int m = 0; m < E / 2; m++) s[m] = f2_fma<PACKED>(k[m], ww, f2_mul<PACKED>(gg, s[m]));
}
// s <- s + w k
template <int E, bool PACKED>
__device__ __forceinline__ void ls_add(f2 (&s)[E / 2], const f2 (&k)[E / 2], float w) {
  const f2 ww = f2_make(w, w);
#pragma unroll
  for (int m = 0; m < E / 2; m++) s[m] = f2_fma<PACKED>(k[m], ww, s[m]);
}
template <int E, int X>
__device__ __forceinline__ void ls_row(f2 (&r)[E / 2], const float* row, int x) {
#pragma unroll
  for (int m = 0; m < E / 4; m++) {
    const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(row + 4 * X * m + 4 * x);
    r[2 * m] = t.x;
    r[2 * m + 1] = t.y;
  }
}

__device__ __forceinline__ void ls_cp16(float* smem, const float* gmem, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem),
               "r"(there ? 16 : 0));
}
__device__ __forceinline__ void ls_cp4(float* smem, const float* gmem, bool there) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem),
               "r"(there ? 4 : 0));
}

// X lanes that hold X partial sums each (acc[0 .. X - 1]) add them up: after the step with distance o a lane keeps the o sums of
// the half that its bit o of x names, and lane x ends with sum x -- the same tree of additions for every sum.
template <int X>
__device__ __forceinline__ float ls_reduce(float (&acc)[X], int x) {
#pragma unroll
  for (int o = X / 2; o > 0; o >>= 1) {
    const bool upper = x & o;
#pragma unroll
    for (int i = 0; i < o; i++) {
      const float send = upper ? acc[i] : acc[i + o], keep = upper ? acc[i + o] : acc[i];
      acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return acc[0];
}

#define LS_COEF 12            // numbers per (token, head) of the delta rule's runs
// What a stage of shared memory holds of LS_GROUP tokens: q, k [LS_GROUP][DP], v [LS_GROUP][COLS] and the decays [LS_GROUP], or
// with the delta rule its coefficients [LS_GROUP][LS_COEF].
template <int DP, bool DELTA, int COLS>
struct LsStage {
  static constexpr int Q = 0, K = LS_GROUP * DP, V = K + LS_GROUP * DP, G = V + LS_GROUP * COLS,
                       FLOATS = G + LS_GROUP * (DELTA ? LS_COEF : 1);
};

// Starts the copies of the tokens tb .. tb + LS_GROUP - 1 of a portion that ends at t1.  Places past its end hold q = k = v = 0, a
// decay of 1 and coefficients of 0 (with 1 for the decays among them), which leave the state as it is.
template <int DP, bool DELTA, int COLS, int THREADS>
__device__ __forceinline__ void ls_fetch(const LinearScan& a, float* st, int tb, int t1, int h, int gk, int j0) {
  using L = LsStage<DP, DELTA, COLS>;
  const int tid = threadIdx.x;
#pragma unroll
  for (int e = tid; e < LS_GROUP * (DP / 4); e += THREADS) {
    const int tt = e / (DP / 4), c = (e - tt * (DP / 4)) * 4;
    const bool there = tb + tt < t1;
    const size_t src = there ? ((size_t)(tb + tt) * a.G + gk) * DP + c : 0;
    ls_cp16(st + L::Q + tt * DP + c, a.q + src, there);
    ls_cp16(st + L::K + tt * DP + c, a.k + src, there);
  }
#pragma unroll
  for (int e = tid; e < LS_GROUP * COLS; e += THREADS) {
    const int tt = e / COLS, c = e - tt * COLS;
    const bool there = tb + tt < t1 && j0 + c < a.dv;
    if (!DELTA && a.nrm && j0 + c == a.dv) st[L::V + e] = tb + tt < t1 ? 1.0f : 0.0f;
    else ls_cp4(st + L::V + e, there ? a.v + (size_t)(tb + tt) * a.ldv + (size_t)h * a.dv + j0 + c : a.v, there);
  }
  if (DELTA) {
    if (tid < LS_GROUP * (LS_COEF / 4)) {
      const int tt = tid / (LS_COEF / 4), c = tid - tt * (LS_COEF / 4);
      float* dst = st + L::G + tt * LS_COEF + 4 * c;
      if (tb + tt < t1) ls_cp16(dst, a.coef + ((size_t)(tb + tt) * a.H + h) * LS_COEF + 4 * c, true);
      else *reinterpret_cast<float4*>(dst) = c == 2 ? make_float4(a.coef[((size_t)(t1 - 1) * a.H + h) * LS_COEF + 8], 1.f, 0.f, 0.f)
                                                    : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else if (tid < LS_GROUP) {
    if (tb + tid < t1) ls_cp4(st + L::G + tid, a.g + (a.g_ld ? (size_t)(tb + tid) * a.g_ld : 0) + h, true);
    else st[L::G + tid] = 1.0f;
  }
  asm volatile("cp.async.commit_group;\n" ::);
}

// Without the delta rule: grid (ceil(dv / COLS), H, requests); eight neighbouring lanes share CPT neighbouring value columns (a
// thread reads its part of k and q once for all of them); token by token.  out float32 [T, H * dv] dense.
template <int DP, int COLS, int CPT>
__global__ void __launch_bounds__(8 * COLS / CPT)
linear_scan_kernel(LinearScan a, float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  using L = LsStage<DP, false, COLS>;
  constexpr int THREADS = 8 * COLS / CPT, E = DP / 8, RUN = 8 / CPT;
  extern __shared__ __align__(16) float ls_sm[];      // two stages
  const int tid = threadIdx.x, x = tid & 7, jl = (tid >> 3) * CPT;
  // a CTA that holds nothing but a normaliser has little to do: those come last, beside others
  int h = blockIdx.y, piece = blockIdx.x;
  if (a.nrm && a.dv % COLS == 0) {
    const int b = h * gridDim.x + piece, full = gridDim.x - 1;
    h = b < a.H * full ? b / full : b - a.H * full;
    piece = b < a.H * full ? b - h * full : full;
  }
  const int req = blockIdx.z, j0 = piece * COLS, j = j0 + jl;
  const int gk = h / (a.H / a.G), d = a.d, dv = a.dv, nc = dv + a.nrm;
  const int t0 = a.cu_tokens[req], t1 = a.cu_tokens[req + 1];
  if (t0 >= t1) return;
  float* S = a.state + (size_t)a.slots[req] * a.state_stride + a.s_off + (size_t)h * nc * d;
  ls_fetch<DP, false, COLS, THREADS>(a, ls_sm, t0, t1, h, gk, j0);
  const bool busy = j0 + (tid >> 5) * 4 * CPT < nc;   // whether this warp has a column at all
  f2 s[CPT][E / 2];
#pragma unroll
  for (int c = 0; c < CPT; c++) ls_load_state<E, 8>(s[c], S + (size_t)(j + c < nc ? j + c : 0) * d, x, d, j + c < nc, a.vec);
  int stage = 0;
  for (int tb = t0; tb < t1; tb += LS_GROUP, stage ^= 1) {
    if (tb + LS_GROUP < t1) {
      ls_fetch<DP, false, COLS, THREADS>(a, ls_sm + (stage ^ 1) * L::FLOATS, tb + LS_GROUP, t1, h, gk, j0);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    const float* st = ls_sm + stage * L::FLOATS;
    const int nt = busy ? min(LS_GROUP, t1 - tb) : 0;
    for (int b = 0; b < nt; b += RUN) {
      float acc[8];                                   // token b + p, column jl + c: this thread's share at CPT p + c
#pragma unroll
      for (int p = 0; p < RUN; p++) {
        const int tt = b + p;
        f2 kr[E / 2], qr[E / 2];
        ls_row<E, 8>(kr, st + L::K + tt * DP, x);
        ls_row<E, 8>(qr, st + L::Q + tt * DP, x);
        const float g = st[L::G + tt];
#pragma unroll
        for (int c = 0; c < CPT; c++) {
          ls_move<E, false>(s[c], kr, st[L::V + tt * COLS + jl + c], g);
          acc[CPT * p + c] = ls_dot<E, false>(s[c], qr);
        }
      }
      const float o = ls_reduce<8>(acc, x);
      const int tt = b + x / CPT, c = j + x % CPT;
      if (tt < nt && c < dv) out[(size_t)(tb + tt) * a.H * dv + (size_t)h * dv + c] = o;
      else if (tt < nt && c < nc) a.nq[(size_t)(tb + tt) * a.H + h] = o;
    }
    __syncthreads();                                  // this stage is overwritten by the next turn's fetch
  }
  if (!a.write_state) return;
#pragma unroll
  for (int c = 0; c < CPT; c++)
    if (j + c < nc) ls_store_state<E, 8>(s[c], S + (size_t)(j + c) * d, x, d, a.vec);
}

// The delta rule in runs of four tokens.  With S0 the state before a run, G_p = g_0 .. g_p and d(s, p) = g_(s+1) .. g_p,
//   x_p = beta_p (v_p - G_p S0^T k_p - sum_(s < p) d(s, p) (k_s . k_p) x_s)
//   o_p = G_p S0^T q_p + sum_(s <= p) d(s, p) (k_s . q_p) x_s;        S <- G_3 S0 + sum_s d(s, 3) k_s x_s^T
// which is the rule token by token written out: the four tokens' products with S0 do not wait for one another, only the
// small triangular system is solved in order.  A run starts at a multiple of four tokens of the portion.
//
// Every number in these sums that does not depend on the state, per (token, head), in ``coef`` [T, H, LS_COEF]: with p the
// token's place in its run,
//   beta d(s, p) (k_s . k_p) for s < p [0 .. 2];  beta G_p [3];  d(s, p) (k_s . q_p) for s <= p [4 .. 7];  G_p [8];
//   d(p, the run's last token) [9];  beta [10]          (zero for later s)
// A warp per (token, query/key head): the dot products once, then the numbers of the value heads that share it.
template <int DP>
__global__ void __launch_bounds__(256)
linear_coef_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ g, int g_ld,
                   const float* __restrict__ beta, int T, int H, int G, const int* __restrict__ token_req,
                   const int* __restrict__ cu_tokens, float* __restrict__ coef) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= (long long)T * G) return;
  const int t = (int)(item / G), gk = (int)(item - (long long)t * G);
  const int r = token_req[t], p = (t - cu_tokens[r]) & 3, last = min(3, p + cu_tokens[r + 1] - 1 - t);
  constexpr int N = DP / 32;
  float kt[N], qt[N];
#pragma unroll
  for (int i = 0; i < N; i++) {
    kt[i] = k[item * DP + lane + 32 * i];
    qt[i] = q[item * DP + lane + 32 * i];
  }
  float kk[4], kq[4];
#pragma unroll
  for (int s = 0; s < 4; s++) {
    kk[s] = kq[s] = 0.f;
    if (s > p) continue;                              // the same for the whole warp
    const float* ks = k + ((size_t)(t - p + s) * G + gk) * DP;
#pragma unroll
    for (int i = 0; i < N; i++) {
      const float y = ks[lane + 32 * i];
      kk[s] = fmaf(y, kt[i], kk[s]);
      kq[s] = fmaf(y, qt[i], kq[s]);
    }
    kk[s] = warp_sum(kk[s]);
    kq[s] = warp_sum(kq[s]);
  }
  const int per = H / G;
  for (int i = lane; i < per; i += 32) {
    const int h = gk * per + i;
    auto decay = [&](int s) { return g[(g_ld ? (size_t)(t - p + s) * g_ld : 0) + h]; };
    const float b = beta[(size_t)t * H + h];
    float A[4] = {0.f, 0.f, 0.f, 0.f}, B[4] = {0.f, 0.f, 0.f, 0.f}, dec = 1.f, to_end = 1.f;
#pragma unroll
    for (int s = 3; s >= 0; s--) {
      if (s > p) continue;
      if (s < p) {
        dec *= decay(s + 1);
        A[s] = b * dec * kk[s];
      }
      B[s] = dec * kq[s];
    }
    dec *= decay(0);
    for (int s = p + 1; s <= last; s++) to_end *= decay(s);
    float4* c = reinterpret_cast<float4*>(coef + ((size_t)t * H + h) * LS_COEF);
    c[0] = make_float4(A[0], A[1], A[2], b * dec);
    c[1] = make_float4(B[0], B[1], B[2], B[3]);
    c[2] = make_float4(dec, to_end, b, 0.f);
  }
}

// grid (ceil(dv / COLS), H, requests), 8 COLS threads: X = 8 CPT neighbouring lanes share CPT neighbouring value columns, so that a
// run's 4 CPT products with k and 4 CPT with q are X sums over X lanes: one exchange adds all of them up.
template <int DP, int COLS, int CPT>
__global__ void __launch_bounds__(8 * COLS)
linear_delta_kernel(LinearScan a, float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  using L = LsStage<DP, true, COLS>;
  constexpr int THREADS = 8 * COLS, X = 8 * CPT, E = DP / X;
  static_assert(E % 4 == 0, "a lane takes whole pieces of four elements");
  extern __shared__ __align__(16) float ls_sm[];      // two stages
  const int tid = threadIdx.x, x = tid % X, jl = tid / X * CPT;
  const int h = blockIdx.y, req = blockIdx.z, j0 = blockIdx.x * COLS, j = j0 + jl;
  const int gk = h / (a.H / a.G), d = a.d, dv = a.dv;
  const int t0 = a.cu_tokens[req], t1 = a.cu_tokens[req + 1];
  if (t0 >= t1) return;
  float* S = a.state + (size_t)a.slots[req] * a.state_stride + a.s_off + (size_t)h * dv * d;
  ls_fetch<DP, true, COLS, THREADS>(a, ls_sm, t0, t1, h, gk, j0);
  f2 s[CPT][E / 2];
#pragma unroll
  for (int c = 0; c < CPT; c++) ls_load_state<E, X>(s[c], S + (size_t)(j + c < dv ? j + c : 0) * d, x, d, j + c < dv, a.vec);
  // after the exchange: lane x has the product with k (first half) or q (second half) of token xp of a run and column xc
  const int xp = x / CPT & 3, xc = x % CPT;
  const bool with_q = x >= 4 * CPT;
  int stage = 0;
  for (int tb = t0; tb < t1; tb += LS_GROUP, stage ^= 1) {
    if (tb + LS_GROUP < t1) {
      ls_fetch<DP, true, COLS, THREADS>(a, ls_sm + (stage ^ 1) * L::FLOATS, tb + LS_GROUP, t1, h, gk, j0);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    const float* st = ls_sm + stage * L::FLOATS;
    const int nt = min(LS_GROUP, t1 - tb);
    for (int b = 0; b < nt; b += 4) {
      f2 kk[4][E / 2];
      float acc[X];
#pragma unroll
      for (int p = 0; p < 4; p++) {
        f2 r[E / 2];
        ls_row<E, X>(kk[p], st + L::K + (b + p) * DP, x);
        ls_row<E, X>(r, st + L::Q + (b + p) * DP, x);
#pragma unroll
        for (int c = 0; c < CPT; c++) {
          acc[p * CPT + c] = ls_dot<E, true>(s[c], kk[p]);
          acc[4 * CPT + p * CPT + c] = ls_dot<E, true>(s[c], r);
        }
      }
      const float4* co = reinterpret_cast<const float4*>(st + L::G + b * LS_COEF);      // three pieces a token
      const float4 mine = co[3 * xp + 2];
      const float sum = ls_reduce<X>(acc, x);
      const float rhs = fmaf(-co[3 * xp].w, sum, mine.z * st[L::V + (b + xp) * COLS + jl + xc]);
      float w[CPT][4];
#pragma unroll
      for (int c = 0; c < CPT; c++)
#pragma unroll
        for (int p = 0; p < 4; p++) w[c][p] = __shfl_sync(0xffffffffu, rhs, p * CPT + c, X);
      const float4 A1 = co[3], A2 = co[6], A3 = co[9];
#pragma unroll
      for (int c = 0; c < CPT; c++) {
        w[c][1] = fmaf(-A1.x, w[c][0], w[c][1]);
        w[c][2] = fmaf(-A2.y, w[c][1], fmaf(-A2.x, w[c][0], w[c][2]));
        w[c][3] = fmaf(-A3.z, w[c][2], fmaf(-A3.y, w[c][1], fmaf(-A3.x, w[c][0], w[c][3])));
      }
      const int tt = b + xp, col = j + xc;
      if (with_q && tt < nt && col < dv) {
        const float4 B = co[3 * xp + 1];
        const bool second = CPT > 1 && xc;            // CPT is 1 or 2
        float o = mine.x * sum;
        o = fmaf(B.x, second ? w[CPT - 1][0] : w[0][0], o);
        o = fmaf(B.y, second ? w[CPT - 1][1] : w[0][1], o);
        o = fmaf(B.z, second ? w[CPT - 1][2] : w[0][2], o);
        o = fmaf(B.w, second ? w[CPT - 1][3] : w[0][3], o);
        out[(size_t)(tb + tt) * a.H * dv + (size_t)h * dv + col] = o;
      }
      const float g3 = co[11].x, e0 = co[2].y, e1 = co[5].y, e2 = co[8].y;      // the run's last token needs no decay
#pragma unroll
      for (int c = 0; c < CPT; c++) {
        ls_move<E, true>(s[c], kk[0], w[c][0] * e0, g3);
        ls_add<E, true>(s[c], kk[1], w[c][1] * e1);
        ls_add<E, true>(s[c], kk[2], w[c][2] * e2);
        ls_add<E, true>(s[c], kk[3], w[c][3]);
      }
    }
    __syncthreads();                                  // this stage is overwritten by the next turn's fetch
  }
  if (!a.write_state) return;
#pragma unroll
  for (int c = 0; c < CPT; c++)
    if (j + c < dv) ls_store_state<E, X>(s[c], S + (size_t)(j + c) * d, x, d, a.vec);
}

// ---------------------------------------------------------------------------------------------------------- finish
struct LinearFinish {
  const float* gate; long long gate_ld;   // float32 logits, head h's at + h * dv; silu or sigmoid (``gate_kind`` 1) is taken here
  const float* norm; int norm_ld;         // [dv] (norm_ld 0) or [H, dv] (norm_ld dv), or null
  float eps, out_scale;
  int gate_kind;
  const float *nq, *low;                  // [T, H]: o is first divided by max(|nq|, low) + LS_NRM_EPS; or null
  void* out; int out_dtype; long long out_stride;
};

// A group of LANES lanes per (token, head).
template <int LANES>
__global__ void __launch_bounds__(256)
linear_finish_kernel(const float* __restrict__ o, int T, int H, int dv, LinearFinish f, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x % LANES;
  long long item = (long long)blockIdx.x * (256 / LANES) + threadIdx.x / LANES;
  const bool there = item < (long long)T * H;         // every lane of a warp takes part in the shuffles
  if (!there) item = 0;
  const int t = (int)(item / H), h = (int)(item - (long long)t * H);
  const float* row = o + (size_t)item * dv;
  const float* gate = f.gate + (size_t)t * f.gate_ld + (size_t)h * dv;
  const size_t dst = (size_t)t * f.out_stride + (size_t)h * dv;
  float ss = 0.f;
  float4 first = make_float4(0.f, 0.f, 0.f, 0.f);     // this lane's first piece stays in registers
  if (vec) {
    for (int i = lane * 4; i < dv; i += LANES * 4) {
      const float4 y = *reinterpret_cast<const float4*>(row + i);
      if (i == lane * 4) first = y;
      ss += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
    }
  } else {
    for (int i = lane; i < dv; i += LANES) { const float y = row[i]; ss = fmaf(y, y, ss); }
  }
#pragma unroll
  for (int s = LANES / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!there) return;
  const float* norm = f.norm ? f.norm + (size_t)h * f.norm_ld : nullptr;
  float c = f.out_scale;
  if (f.nq) {
    const float r = 1.0f / (fmaxf(fabsf(f.nq[item]), f.low[item]) + LS_NRM_EPS);
    ss *= r * r;
    c *= r;
  }
  c /= sqrtf(ss / (float)dv + f.eps);
  if (vec) {
    for (int i = lane * 4; i < dv; i += LANES * 4) {
      const float4 y = i == lane * 4 ? first : *reinterpret_cast<const float4*>(row + i);
      const float4 z = *reinterpret_cast<const float4*>(gate + i);
      float4 n = make_float4(c, c, c, c);
      if (norm) {
        const float4 w = *reinterpret_cast<const float4*>(norm + i);
        n = make_float4(c * w.x, c * w.y, c * w.z, c * w.w);
      }
      const float4 r = make_float4(y.x * n.x * ls_gate(z.x, f.gate_kind), y.y * n.y * ls_gate(z.y, f.gate_kind),
                                   y.z * n.z * ls_gate(z.z, f.gate_kind), y.w * n.w * ls_gate(z.w, f.gate_kind));
      if (f.out_dtype == QD_F32) {
        *reinterpret_cast<float4*>(reinterpret_cast<float*>(f.out) + dst + i) = r;
      } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(r.x, r.y), hi = __floats2bfloat162_rn(r.z, r.w);
        uint2 raw;
        raw.x = *reinterpret_cast<unsigned*>(&lo);
        raw.y = *reinterpret_cast<unsigned*>(&hi);
        *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(f.out) + dst + i) = raw;
      }
    }
    return;
  }
  for (int i = lane; i < dv; i += LANES)
    ls_st(f.out, f.out_dtype, dst + i, row[i] * c * (norm ? norm[i] : 1.0f) * ls_gate(gate[i], f.gate_kind));
}

// ------------------------------------------------------------------------------------------------------------ step
// grid (H, requests), 4 * (columns at a time) threads, at most LS_STEP_THREADS: four neighbouring lanes to a value column.
// Request r's token is token r.
#define LS_STEP_THREADS(DP) ((DP) > 128 ? 256 : 512)

// A lane's elements of a row of q or k: padded rows, or (``raw``) rows of d numbers where they stand.
template <int E>
__device__ __forceinline__ void ls_step_row(f2 (&r)[E / 2], const float* row, int x, int d, int raw, int vec, float scale) {
  if (!raw) {
    ls_row<E, 4>(r, row, x);
    return;
  }
  ls_load_state<E, 4>(r, row, x, d, true, vec);
  const f2 c = f2_make(scale, scale);
#pragma unroll
  for (int m = 0; m < E / 2; m++) r[m] = f2_mul<false>(r[m], c);
}

template <int DP, bool DELTA>
__global__ void __launch_bounds__(LS_STEP_THREADS(DP))
linear_step_kernel(LinearScan a, LinearFinish f, ExpGates eg) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int E = DP / 4;
  extern __shared__ float st_sm[];                    // [dv + nrm] outputs, then 40 of scratch
  const int tid = threadIdx.x, x = tid & 3, jl = tid >> 2, cols = blockDim.x >> 2;
  const int h = blockIdx.x, t = blockIdx.y, d = a.d, dv = a.dv, nc = dv + a.nrm, gk = h / (a.H / a.G);
  float* kept = a.state + (size_t)a.slots[t] * a.state_stride;
  float* S = kept + a.s_off + (size_t)h * nc * d;
  const long long q_ld = a.raw ? a.q_ld : (long long)a.G * DP;
  const float* kr = a.k + (size_t)t * q_ld + (size_t)gk * (a.raw ? d : DP);
  const float* qr = a.q + (size_t)t * q_ld + (size_t)gk * (a.raw ? d : DP);
  const int qvec = a.vec && q_ld % 4 == 0 && !(((uintptr_t)a.q | (uintptr_t)a.k) & 15);
  float g, in = 1.f, m = 0.f;
  if (!DELTA && eg.on) {
    float i, lf;
    exp_gate_logs(eg, eg.u[(size_t)t * eg.ld + eg.i_off + h], eg.u[(size_t)t * eg.ld + eg.f_off + h], h, i, lf);
    const float m0 = kept[eg.m_off + h];
    m = fmaxf(lf + m0, i);
    g = expf(lf + (m0 - m));
    in = expf(i - m);
  } else {
    g = a.g[(a.g_ld ? (size_t)t * a.g_ld : 0) + h];
  }
  const float beta = DELTA ? a.beta[(size_t)t * a.H + h] : 0.f;
  float ss = 0.f;
  for (int j0 = 0; j0 < nc; j0 += cols) {             // every thread takes every turn: the shuffles need them all
    const int j = j0 + jl;
    const bool live = j < nc;
    float* col = S + (size_t)(live ? j : 0) * d;
    f2 s[E / 2];
    ls_load_state<E, 4>(s, col, x, d, live, a.vec);
    float w = j < dv ? a.v[(size_t)t * a.ldv + (size_t)h * dv + j] : live ? 1.f : 0.f;
    f2 r[E / 2];
    ls_step_row<E>(r, kr, x, d, a.raw, qvec, a.k_scale);
    if (DELTA) {
      float dot = ls_dot<E, false>(s, r);
      dot += __shfl_xor_sync(0xffffffffu, dot, 2);
      dot += __shfl_xor_sync(0xffffffffu, dot, 1);
      w = beta * fmaf(-g, dot, w);
    } else {
      w *= in;
    }
    ls_move<E, false>(s, r, w, g);
    ls_step_row<E>(r, qr, x, d, a.raw, qvec, a.q_scale);
    float o = ls_dot<E, false>(s, r);
    o += __shfl_xor_sync(0xffffffffu, o, 2);
    o += __shfl_xor_sync(0xffffffffu, o, 1);
    if (live && x == 0) {
      st_sm[j] = o;
      if (j < dv) ss = fmaf(o, o, ss);
    }
    if (a.write_state && live) ls_store_state<E, 4>(s, col, x, d, a.vec);
  }
  ss = block_sum(ss, st_sm + nc);                     // meets the writes of st_sm and every thread's read of the maximum, too
  float c = f.out_scale;
  if (a.nrm) {
    const float r = 1.0f / (fmaxf(fabsf(st_sm[dv]), expf(-m)) + LS_NRM_EPS);
    ss *= r * r;
    c *= r;
  }
  c /= sqrtf(ss / (float)dv + f.eps);
  if (!DELTA && eg.on && a.write_state && tid == 0) kept[eg.m_off + h] = m;
  const float* gate = f.gate + (size_t)t * f.gate_ld + (size_t)h * dv;
  const float* norm = f.norm ? f.norm + (size_t)h * f.norm_ld : nullptr;
  for (int i = tid; i < dv; i += blockDim.x)
    ls_st(f.out, f.out_dtype, (size_t)t * f.out_stride + (size_t)h * dv + i,
          st_sm[i] * c * (norm ? norm[i] : 1.0f) * ls_gate(gate[i], f.gate_kind));
}

// ------------------------------------------------------------------------------------------------------- launchers
// q, k float32 [T, G, DP], DP the padded head size: the smallest of 32, 64, 96, 128, 256 that holds d; v rows
// ``ldv`` apart; g float32 [T, H] (g_ld = H) or [H] (g_ld = 0); beta float32 [T, H]: the delta rule, or null;
// state float32 rows ``state_stride`` apart, the heads' matrices [H, dv, d] at ``s_off``; o_buf float32 [T, H * dv]
// (unused when every request brings one token); coef float32 [T, H, LS_COEF] of scratch for the delta rule (unused then, too);
// gate float32 rows ``gate_ld`` apart; norm float32 [dv] (norm_ld 0) or [H, dv] (norm_ld dv), or null; gate_kind 0 silu, 1 sigmoid.
// ``nrm``: exponential gates.  S is [H, dv + 1, d] at ``s_off``, the maxima at ``m_off``; portions: nq scratch [T, H], g, low and k
// as ``qd_linear_exp_gates`` and ``qd_linear_prep`` made them; single tokens: g unused, the logits are columns i_off, f_off of u.
// ``raw`` (single tokens): q and k are rows of G * d numbers ``q_ld`` apart that q_scale and k_scale still multiply.
extern "C" int qd_linear_scan(const float* q, const float* k, const float* v, long long ldv, const float* g, int g_ld,
                              const float* beta, int T, int n_requests, int H, int G, int d, int dv, int DP,
                              float* state, long long state_stride, long long s_off, const int* cu_tokens,
                              const int* slots, int write_state, float* o_buf, const float* gate, long long gate_ld,
                              const float* norm, float eps, float out_scale, void* out, int out_dtype,
                              long long out_stride, const int* token_req, float* coef, int norm_ld, int gate_kind, int nrm,
                              float* nq, const float* low, const float* u, long long u_ld, int i_off, int f_off,
                              const float* ib, const float* fb, float cap, long long m_off, int raw, long long q_ld,
                              float q_scale, float k_scale, cudaStream_t stream) {
  if (T <= 0 || n_requests <= 0) return 0;
  if (H <= 0 || H > 65535 || n_requests > 65535 || G <= 0 || H % G || d <= 0 || dv <= 0 || dv > 8192 || d > DP ||
      !state || !gate || (g_ld && g_ld != H) || (beta && T != n_requests && (!coef || ((uintptr_t)coef & 15))) || (out_dtype != QD_F32 && out_dtype != QD_BF16))
    return QD_ERR_UNSUPPORTED;
  const bool single = T == n_requests;                // every request has at least one token
  if (!single && !o_buf) return QD_ERR_UNSUPPORTED;
  if (nrm && (beta || G != H || (single ? !u || !ib || !fb || !(cap > 0.f) : !nq || !low))) return QD_ERR_UNSUPPORTED;
  if (raw ? !single : (((uintptr_t)q | (uintptr_t)k) & 15) != 0) return QD_ERR_UNSUPPORTED;
  if (!g && !(nrm && single)) return QD_ERR_UNSUPPORTED;
  nrm = nrm ? 1 : 0;
  const int nc = dv + nrm;
  const int vec = d % 4 == 0 && state_stride % 4 == 0 && s_off % 4 == 0 && !((uintptr_t)state & 15);
  const LinearScan a = {q, k, v, ldv, g, g_ld, beta, coef, H, G, d, dv, state, state_stride, s_off, vec, cu_tokens, slots,
                        write_state, nrm, nq, raw, q_ld, q_scale, k_scale};
  const LinearFinish f = {gate, gate_ld, norm, norm_ld, eps, out_scale, gate_kind, nrm ? nq : nullptr, low, out, out_dtype,
                          out_stride};
  const ExpGates eg = {u, u_ld, i_off, f_off, ib, fb, cap, m_off, nrm};
  // as many columns at a time as make the turns even
  const int most = LS_STEP_THREADS(DP) / 4, turns = (nc + most - 1) / most, cols = ((nc + turns - 1) / turns + 7) / 8 * 8;
  const size_t step_smem = ((size_t)nc + 40) * sizeof(float);
  // few heads: half as many columns to a CTA, so that more multiprocessors work (the CTA of a normaliser's single column
  // costs next to nothing)
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  }
  const bool narrow = (long long)((dv + 31) / 32) * H * n_requests * 2 <= sms + sms / 8;
#define LS_LAUNCH(KERNEL, COLS, THREADS, FLOATS)                                                                     \
  do {                                                                                                                \
    const size_t smem = (size_t)(FLOATS) * sizeof(float);                                                             \
    static bool raised = false;                                                                                       \
    if (!raised && smem > 48 * 1024) {                                                                                \
      cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                           \
      raised = true;                                                                                                  \
    }                                                                                                                 \
    /* The scan's CTAs are few and long: launched while the kernel before them still runs they would crowd onto the   \
       multiprocessors that become free first. */                                                                     \
    qd_plain_next_launch = true;                                                                                      \
    qd_launch(KERNEL, dim3((nc + COLS - 1) / COLS, H, n_requests), dim3(THREADS), smem, stream, a, o_buf);             \
  } while (0)
#define LS_DELTA(DP)                                                                                                  \
  do {                                                                                                                \
    if (single) {                                                                                                     \
      qd_launch(linear_step_kernel<DP, true>, dim3(H, n_requests), dim3(4 * cols), step_smem, stream, a, f, eg);          \
      break;                                                                                                          \
    }                                                                                                                 \
    qd_launch(linear_coef_kernel<DP>, dim3((unsigned)(((long long)T * G + 7) / 8)), dim3(256), 0, stream, q, k, g, g_ld, \
              beta, T, H, G, token_req, cu_tokens, coef);                                                             \
    constexpr int CPT = DP <= 96 ? 1 : 2;                                                                             \
    if (narrow) LS_LAUNCH((linear_delta_kernel<DP, 16, CPT>), 16, 128, (2 * LsStage<DP, true, 16>::FLOATS));           \
    else LS_LAUNCH((linear_delta_kernel<DP, 32, CPT>), 32, 256, (2 * LsStage<DP, true, 32>::FLOATS));                  \
  } while (0)
#define LS_PLAIN(DP)                                                                                                  \
  do {                                                                                                                \
    if (single) qd_launch(linear_step_kernel<DP, false>, dim3(H, n_requests), dim3(4 * cols), step_smem, stream, a, f, eg); \
    else if (narrow) LS_LAUNCH((linear_scan_kernel<DP, 16, 1>), 16, 128, (2 * LsStage<DP, false, 16>::FLOATS));        \
    else LS_LAUNCH((linear_scan_kernel<DP, 32, 2>), 32, 128, (2 * LsStage<DP, false, 32>::FLOATS));                    \
  } while (0)
#define LS_GO(DP) do { if (beta) LS_DELTA(DP); else LS_PLAIN(DP); } while (0)
  switch (DP) {
    case 32: LS_GO(32); break;
    case 64: LS_GO(64); break;
    case 96: LS_GO(96); break;
    case 128: LS_GO(128); break;
    case 256: LS_GO(256); break;
    default: return QD_ERR_UNSUPPORTED;
  }
#undef LS_GO
#undef LS_DELTA
#undef LS_PLAIN
#undef LS_LAUNCH
  if (!single) {
    const int fvec = dv % 4 == 0 && gate_ld % 4 == 0 && out_stride % 4 == 0 &&
                     !(((uintptr_t)o_buf | (uintptr_t)gate | (uintptr_t)norm) & 15) &&
                     !((uintptr_t)out & (out_dtype == QD_F32 ? 15 : 7));
    const long long items = (long long)T * H;
    if (dv <= 64)
      qd_launch(linear_finish_kernel<16>, dim3((unsigned)((items + 15) / 16)), dim3(256), 0, stream, (const float*)o_buf, T, H, dv, f, fvec);
    else
      qd_launch(linear_finish_kernel<32>, dim3((unsigned)((items + 7) / 8)), dim3(256), 0, stream, (const float*)o_buf, T, H, dv, f, fvec);
  }
  return qd_last_error();
}
