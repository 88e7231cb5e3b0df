// RMS norms in groups, before and after a branch, as one launch between two branches:
//
//   y = sum of the branch output's partial sums (+ a bias per channel)
//   x[s] += G(y; post_w, post_eps, post_groups)          (without post_w: x[s] += y)
//   out[r] = G(x[s]; pre_w, pre_eps, pre_groups), s = rows[r] (or r);  without pre_w out[r] = x[s], and without out nothing is written
//
// G(v; w, eps, n): v is cut into n equal consecutive parts, every part is divided by its own sqrt(mean(part^2) + eps),
// and the whole is multiplied by w.  float32 throughout; one CTA per row; the order of a part's sum depends on the
// sizes only.
#include "common.cuh"

struct GroupNorm {
  float* x;
  const void* delta; int delta_dtype, n_parts; size_t part_stride;      // null: nothing is pending
  const float* delta_bias;
  const float* post_w; float post_eps; int post_groups;
  const float* pre_w; float pre_eps; int pre_groups;
  void* out; int out_dtype;
  const int* rows;
  int D, write_back;
};

// f[g] = 1 / sqrt(mean over group g + eps) from ``n`` partial sums of squares in ``sq`` (n / groups of them per group,
// ``part`` elements each group).  Warps share the groups: several warps to a group when there are few groups.
// scratch: max(groups, warps) floats.
__device__ __forceinline__ void group_factors(const float* sq, int n, int groups, int part, float eps, float* scratch,
                                              float* f) {
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wpg = groups < warps ? warps / groups : 1, per = n / groups, sub = warp % wpg;
  __syncthreads();
  for (int g = warp / wpg; g < groups; g += warps / wpg) {
    float s = 0.f;
    for (int i = sub * 32 + lane; i < per; i += 32 * wpg) s += sq[(size_t)g * per + i];
    s = warp_sum(s);
    if (lane == 0) scratch[g * wpg + sub] = s;
  }
  __syncthreads();
  for (int g = threadIdx.x; g < groups; g += blockDim.x) {
    float s = 0.f;
    for (int i = 0; i < wpg; i++) s += scratch[g * wpg + i];
    f[g] = 1.0f / sqrtf(s / (float)part + eps);
  }
  __syncthreads();
}

// Four neighbouring elements of the branch's output: its partial sums added up, and its bias.
__device__ __forceinline__ float4 delta4(const GroupNorm& a, size_t s, int i, float4 bias) {
  float4 d;
  if (a.delta_dtype == QD_F32) {
    const float4* dp = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(a.delta) + s * a.D) + i;
    d = *dp;
    for (int p = 1; p < a.n_parts; p++) {
      const float4 e = dp[p * (a.part_stride >> 2)];
      d.x += e.x; d.y += e.y; d.z += e.z; d.w += e.w;
    }
  } else {
    const uint2 raw = reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(a.delta) + s * a.D)[i];
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x);
    const __nv_bfloat162 hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    d = make_float4(__low2float(lo), __high2float(lo), __low2float(hi), __high2float(hi));
  }
  return make_float4(d.x + bias.x, d.y + bias.y, d.z + bias.z, d.w + bias.w);
}
__device__ __forceinline__ void out4(const GroupNorm& a, size_t r, int i, float4 o) {
  if (a.out_dtype == QD_F32) {
    reinterpret_cast<float4*>(reinterpret_cast<float*>(a.out) + r * a.D)[i] = o;
    return;
  }
  __nv_bfloat162 lo = __floats2bfloat162_rn(o.x, o.y), hi = __floats2bfloat162_rn(o.z, o.w);
  uint2 raw;
  raw.x = *reinterpret_cast<unsigned*>(&lo);
  raw.y = *reinterpret_cast<unsigned*>(&hi);
  reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(a.out) + r * a.D)[i] = raw;
}
__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// ------------------------------------------------------------------------------------- parts of whole warps
// Every part of D a multiple of 128 elements: the 32 float4 that a warp holds at one turn lie in one part, so a norm costs
// one meeting of the CTA -- every warp leaves its sum, and adds up its part's sums itself.
template <int VPT, int MAX_THREADS>
__global__ void __launch_bounds__(MAX_THREADS)
group_add_norm_warp_kernel(GroupNorm a) {
  pdl_launch_dependents();
  extern __shared__ float gn_sm[];                    // [D / 128] sums of each norm
  const int n4 = a.D >> 2, lane = threadIdx.x & 31;
  float4 wp[VPT], wn[VPT], bias[VPT], v[VPT], xv[VPT];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int q = 0; q < VPT; q++) {                     // no kernel of a step writes these
    const int i = threadIdx.x + q * blockDim.x;
    wp[q] = (a.post_w && i < n4) ? reinterpret_cast<const float4*>(a.post_w)[i] : zero;
    wn[q] = (a.pre_w && i < n4) ? reinterpret_cast<const float4*>(a.pre_w)[i] : zero;
    bias[q] = (a.delta_bias && i < n4) ? reinterpret_cast<const float4*>(a.delta_bias)[i] : zero;
  }
  pdl_wait();
  const int r = blockIdx.x;
  const size_t s = a.rows ? (size_t)a.rows[r] : (size_t)r;
  float4* xr = reinterpret_cast<float4*>(a.x + s * a.D);
  float* sums = gn_sm;
  // 1 / sqrt(mean over the part of this warp's float4 ``i`` + eps)
  auto factor = [&](int i, int part4, float eps) {
    const int g0 = i / part4 * (part4 >> 5);
    float t = 0.f;
    for (int k = lane; k < part4 >> 5; k += 32) t += sums[g0 + k];
    return 1.0f / sqrtf(warp_sum(t) / (float)(4 * part4) + eps);
  };
#pragma unroll
  for (int q = 0; q < VPT; q++) {
    const int i = threadIdx.x + q * blockDim.x;
    xv[q] = v[q] = zero;
    if (i < n4) {
      xv[q] = xr[i];
      if (a.delta) v[q] = delta4(a, s, i, bias[q]);
    }
  }
  if (a.delta && a.post_w) {
#pragma unroll
    for (int q = 0; q < VPT; q++) {
      const int i = threadIdx.x + q * blockDim.x;
      const float t = warp_sum(sq4(v[q]));
      if (lane == 0 && i < n4) sums[i >> 5] = t;
    }
    __syncthreads();
    const int part4 = n4 / a.post_groups;
#pragma unroll
    for (int q = 0; q < VPT; q++) {
      const int i = threadIdx.x + q * blockDim.x;
      if (i >= n4) continue;                          // whole warps: D is a multiple of 128
      const float c = factor(i, part4, a.post_eps);
      v[q] = make_float4(v[q].x * c * wp[q].x, v[q].y * c * wp[q].y, v[q].z * c * wp[q].z, v[q].w * c * wp[q].w);
    }
  }
  sums = gn_sm + (n4 >> 5);
#pragma unroll
  for (int q = 0; q < VPT; q++) {
    const int i = threadIdx.x + q * blockDim.x;
    xv[q].x += v[q].x; xv[q].y += v[q].y; xv[q].z += v[q].z; xv[q].w += v[q].w;
    if (a.delta && a.write_back && i < n4) xr[i] = xv[q];
    if (a.pre_w) {
      const float t = warp_sum(sq4(xv[q]));
      if (lane == 0 && i < n4) sums[i >> 5] = t;
    }
  }
  if (!a.out) return;
  if (!a.pre_w) {                                     // the sum itself, rounded
#pragma unroll
    for (int q = 0; q < VPT; q++) {
      const int i = threadIdx.x + q * blockDim.x;
      if (i < n4) out4(a, (size_t)r, i, xv[q]);
    }
    return;
  }
  __syncthreads();
  const int part4 = n4 / a.pre_groups;
#pragma unroll
  for (int q = 0; q < VPT; q++) {
    const int i = threadIdx.x + q * blockDim.x;
    if (i >= n4) continue;
    const float c = factor(i, part4, a.pre_eps);
    out4(a, (size_t)r, i, make_float4(xv[q].x * c * wn[q].x, xv[q].y * c * wn[q].y, xv[q].z * c * wn[q].z, xv[q].w * c * wn[q].w));
  }
}

// ------------------------------------------------------------------------------------- four elements at a time
// D and the parts multiples of 4, every pointer 16-byte aligned, D <= 4 * VPT * blockDim.
template <int VPT>
__global__ void __launch_bounds__(1024)
group_add_norm_vec_kernel(GroupNorm a) {
  pdl_launch_dependents();
  extern __shared__ float gn_sm[];                    // [D / 4] squares, then scratch, then factors
  const int n4 = a.D >> 2, warps = blockDim.x >> 5;
  const int most = max(max(a.post_groups, a.pre_groups), warps);
  float* sq = gn_sm;
  float* scratch = gn_sm + n4;
  float* f = scratch + most;
  float4 wp[VPT], wn[VPT], bias[VPT], v[VPT];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int q = 0; q < VPT; q++) {                     // no kernel of a step writes these
    const int i = threadIdx.x + q * blockDim.x;
    wp[q] = (a.post_w && i < n4) ? reinterpret_cast<const float4*>(a.post_w)[i] : zero;
    wn[q] = (a.pre_w && i < n4) ? reinterpret_cast<const float4*>(a.pre_w)[i] : zero;
    bias[q] = (a.delta_bias && i < n4) ? reinterpret_cast<const float4*>(a.delta_bias)[i] : zero;
  }
  pdl_wait();
  const int r = blockIdx.x;
  const size_t s = a.rows ? (size_t)a.rows[r] : (size_t)r;
  float4* xr = reinterpret_cast<float4*>(a.x + s * a.D);
  float4 xv[VPT];
#pragma unroll
  for (int q = 0; q < VPT; q++) {
    const int i = threadIdx.x + q * blockDim.x;
    xv[q] = v[q] = zero;
    if (i >= n4) continue;
    xv[q] = xr[i];
    if (!a.delta) continue;
    v[q] = delta4(a, s, i, bias[q]);
    if (a.post_w) sq[i] = sq4(v[q]);
  }
  const int post_part4 = n4 / a.post_groups, pre_part4 = n4 / a.pre_groups;
  if (a.delta && a.post_w) group_factors(sq, n4, a.post_groups, post_part4 * 4, a.post_eps, scratch, f);
#pragma unroll
  for (int q = 0; q < VPT; q++) {
    const int i = threadIdx.x + q * blockDim.x;
    if (i >= n4) continue;
    if (a.delta) {
      if (a.post_w) {
        const float c = f[i / post_part4];
        v[q] = make_float4(v[q].x * c * wp[q].x, v[q].y * c * wp[q].y, v[q].z * c * wp[q].z, v[q].w * c * wp[q].w);
      }
      xv[q].x += v[q].x; xv[q].y += v[q].y; xv[q].z += v[q].z; xv[q].w += v[q].w;
      if (a.write_back) xr[i] = xv[q];
    }
    if (a.pre_w) sq[i] = sq4(xv[q]);
  }
  if (!a.out) return;
  if (!a.pre_w) {
#pragma unroll
    for (int q = 0; q < VPT; q++) {
      const int i = threadIdx.x + q * blockDim.x;
      if (i < n4) out4(a, (size_t)r, i, xv[q]);
    }
    return;
  }
  group_factors(sq, n4, a.pre_groups, pre_part4 * 4, a.pre_eps, scratch, f);
#pragma unroll
  for (int q = 0; q < VPT; q++) {
    const int i = threadIdx.x + q * blockDim.x;
    if (i >= n4) continue;
    const float c = f[i / pre_part4];
    out4(a, (size_t)r, i, make_float4(xv[q].x * c * wn[q].x, xv[q].y * c * wn[q].y, xv[q].z * c * wn[q].z, xv[q].w * c * wn[q].w));
  }
}

// ------------------------------------------------------------------------------------------------ any sizes
__global__ void __launch_bounds__(256)
group_add_norm_kernel(GroupNorm a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float gn_sm[];                    // [D] values, [D] squares, then scratch, then factors
  const int D = a.D, warps = blockDim.x >> 5;
  const int most = max(max(a.post_groups, a.pre_groups), warps);
  float *v = gn_sm, *sq = v + D, *scratch = sq + D, *f = scratch + most;
  const int r = blockIdx.x;
  const size_t s = a.rows ? (size_t)a.rows[r] : (size_t)r;
  float* xr = a.x + s * D;
  if (a.delta)
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
      float d;
      if (a.delta_dtype == QD_F32) {
        const float* dp = reinterpret_cast<const float*>(a.delta) + s * D + i;
        d = dp[0];
        for (int p = 1; p < a.n_parts; p++) d += dp[p * a.part_stride];
      } else {
        d = __bfloat162float(reinterpret_cast<const bf16*>(a.delta)[s * D + i]);
      }
      if (a.delta_bias) d += a.delta_bias[i];
      v[i] = d;
      sq[i] = d * d;
    }
  const int post_part = D / a.post_groups, pre_part = D / a.pre_groups;
  if (a.delta && a.post_w) group_factors(sq, D, a.post_groups, post_part, a.post_eps, scratch, f);
  for (int i = threadIdx.x; i < D; i += blockDim.x) {           // a thread meets the elements it wrote above
    float x = xr[i];
    if (a.delta) {
      x += a.post_w ? v[i] * f[i / post_part] * a.post_w[i] : v[i];
      if (a.write_back) xr[i] = x;
    }
    v[i] = x;
    sq[i] = x * x;
  }
  if (!a.out) return;
  if (a.pre_w) group_factors(sq, D, a.pre_groups, pre_part, a.pre_eps, scratch, f);
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    const float o = a.pre_w ? v[i] * f[i / pre_part] * a.pre_w[i] : v[i];
    if (a.out_dtype == QD_F32) reinterpret_cast<float*>(a.out)[(size_t)r * D + i] = o;
    else reinterpret_cast<bf16*>(a.out)[(size_t)r * D + i] = __float2bfloat16_rn(o);
  }
}

// x float32 [T, D]; delta [T, D] (``delta_dtype``) or float32 partial sums [n_parts, T, D] ``part_stride`` apart, or null;
// delta_bias float32 [D] or null; post_w / pre_w float32 [D] or null; out [n_rows, D]; rows int32 [n_rows] or null.
extern "C" int qd_group_add_norm(float* x, const void* delta, int delta_dtype, int n_parts, long long part_stride,
                                 const float* delta_bias, const float* post_w, float post_eps, int post_groups,
                                 const float* pre_w, float pre_eps, int pre_groups, void* out, int out_dtype,
                                 const int* rows, int n_rows, int D, int write_back, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (!post_w) post_groups = 1;
  if (!pre_w) pre_groups = 1;
  if (D <= 0 || post_groups < 1 || pre_groups < 1 || D % post_groups || D % pre_groups || n_parts < 1 || (pre_w && !out) ||
      (delta && delta_dtype != QD_F32 && (delta_dtype != QD_BF16 || n_parts != 1)) ||
      (out && out_dtype != QD_F32 && out_dtype != QD_BF16))
    return QD_ERR_UNSUPPORTED;
  const GroupNorm a = {x, delta, delta_dtype, n_parts, (size_t)part_stride, delta_bias, post_w, post_eps, post_groups,
                       pre_w, pre_eps, pre_groups, out, out_dtype, rows, D, write_back};
  const int groups = post_groups > pre_groups ? post_groups : pre_groups;
  const uintptr_t all = (uintptr_t)x | (uintptr_t)delta | (uintptr_t)delta_bias | (uintptr_t)post_w | (uintptr_t)pre_w |
                        (uintptr_t)out;
  if ((D / post_groups) % 4 == 0 && (D / pre_groups) % 4 == 0 && !(all & 15) && part_stride % 4 == 0 && D <= 16384) {
    const int n4 = D / 4;
    if ((D / post_groups) % 128 == 0 && (D / pre_groups) % 128 == 0) {
      const size_t smem = (size_t)2 * (n4 / 32) * sizeof(float);
      // few rows: one piece a thread; many rows: two or four, so that more rows are under way
      if (n4 <= 256) qd_launch(group_add_norm_warp_kernel<1, 256>, dim3(n_rows), dim3(n4), smem, stream, a);
      else if (n4 <= 512 && n_rows > 128)
        qd_launch(group_add_norm_warp_kernel<2, 256>, dim3(n_rows), dim3((n4 / 2 + 31) / 32 * 32), smem, stream, a);
      else if (n4 <= 1024 && n_rows > 128)
        qd_launch(group_add_norm_warp_kernel<4, 256>, dim3(n_rows), dim3((n4 / 4 + 31) / 32 * 32), smem, stream, a);
      else if (n4 <= 1024) qd_launch(group_add_norm_warp_kernel<1, 1024>, dim3(n_rows), dim3(n4), smem, stream, a);
      else if (n4 <= 2048) qd_launch(group_add_norm_warp_kernel<2, 1024>, dim3(n_rows), dim3((n4 / 2 + 31) / 32 * 32), smem, stream, a);
      else qd_launch(group_add_norm_warp_kernel<4, 1024>, dim3(n_rows), dim3((n4 / 4 + 31) / 32 * 32), smem, stream, a);
      return qd_last_error();
    }
    const int threads = n4 < 1024 ? (n4 + 31) / 32 * 32 : 1024;
    const int most = groups > threads / 32 ? groups : threads / 32;
    const size_t smem = ((size_t)n4 + 2 * most) * sizeof(float);          // at most 4,096 * 3 floats
    if (smem > 48 * 1024) return QD_ERR_UNSUPPORTED;
    if (n4 <= threads) qd_launch(group_add_norm_vec_kernel<1>, dim3(n_rows), dim3(threads), smem, stream, a);
    else if (n4 <= 2 * threads) qd_launch(group_add_norm_vec_kernel<2>, dim3(n_rows), dim3(threads), smem, stream, a);
    else qd_launch(group_add_norm_vec_kernel<4>, dim3(n_rows), dim3(threads), smem, stream, a);
    return qd_last_error();
  }
  const int most = groups > 8 ? groups : 8;
  const size_t smem = ((size_t)2 * D + 2 * most) * sizeof(float);
  if (smem > 200 * 1024) return QD_ERR_UNSUPPORTED;
  static size_t raised = 48 * 1024;
  if (smem > raised) {
    cudaFuncSetAttribute(group_add_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    raised = smem;
  }
  qd_launch(group_add_norm_kernel, dim3(n_rows), dim3(256), smem, stream, a);
  return qd_last_error();
}
