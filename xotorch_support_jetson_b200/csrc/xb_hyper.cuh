// The residual stream as n copies of one row (hyper-connections), with the norm that reads it next; n = 1 with no mixing is the
// plain residual sum, so a layer norm without copies runs here too.  Included by xb_hybrid_kernels.cuh.
//
//   x_j <- sum_i mix[i, j] x_i + out[j] y          (all copies at once from the old ones; skipped when there is no y)
//   u    = sum_i rd[i] x_i                          (rd == nullptr: their sum)
//   hn / ha = norm(u)                               (fp32 row / Linear input; either may be nullptr)
// y may carry the part of a feed-forward that hands its input on: y += (sum of same_w[t, 0 .. same_n)) * same[t, :], the rows in the
// type a Linear reads (same may be the very buffer that ha overwrites: a thread reads the channels it writes).
// tokens != nullptr: every copy starts as the token's embedding row (no y).  Everything is fp32.
#pragma once
#include <cooperative_groups.h>

#define HY_MAX_STREAMS 16
struct HyperArgs {
  float* x;                 // [T][n][D]
  int n, D;
  LinOut y;
  const float *mix, *out;   // [n][n] (from, to), [n]; nullptr: the identity / ones
  const float* rd;          // [n]
  const float* nw;          // [D], or one number (nw_mode 2)
  int norm, nw_mode;        // XB_NORM_RMS or XB_NORM_LAYER; weight form as in RowOpArgs
  float eps;
  float* hn;
  void* ha;
  const void* same;         // [T][D] of AT
  const float* same_w;      // row pitch same_ld
  int same_ld, same_n;
  const int* tokens;
  const bf16* emb;
  int V;
  float emb_scale;
};

template <int VEC> struct HyVec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ HyVec<VEC> hy_ldv(const float* p) {
  HyVec<VEC> r;
  if constexpr (VEC == 4) { const float4 a = *reinterpret_cast<const float4*>(p); r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w; }
  else r.v[0] = *p;
  return r;
}
template <int VEC> __device__ __forceinline__ HyVec<VEC> hy_ldv(const bf16* p) {
  HyVec<VEC> r;
  if constexpr (VEC == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = bf2_to_f2(u.x), b = bf2_to_f2(u.y);
    r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
  } else r.v[0] = bf2f(*p);
  return r;
}
template <int VEC> __device__ __forceinline__ void hy_stv(float* p, const HyVec<VEC>& a) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]);
  else *p = a.v[0];
}
template <int VEC> __device__ __forceinline__ void hy_stv(bf16* p, const HyVec<VEC>& a) {
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf2(a.v[0], a.v[1]), f2_to_bf2(a.v[2], a.v[3]));
  else *p = f2bf(a.v[0]);
}

// SM: most copies this instantiation holds in registers.  VEC neighbouring channels per thread (4: D a multiple of 4, y one bf16
// matrix or one fp32 plane with a pitch that is a multiple of 4).  One block per row; dynamic shared memory D floats.
template <typename AT, int NT, int SM, int VEC>
__global__ void __launch_bounds__(NT) hy_hyper_kernel(HyperArgs a) {
  extern __shared__ __align__(16) float row[];
  __shared__ float wm[SM * SM], wo[SM], wr[SM];
  __shared__ float red[32];
  const int n = a.n, D = a.D;
  pdl_launch_dependents();
  const bool branch = a.y.f != nullptr || a.y.h != nullptr;
  for (int i = threadIdx.x; i < SM * SM; i += NT) {
    const int f = i / SM, t = i - f * SM;
    wm[i] = (f < n && t < n) ? (a.mix != nullptr ? a.mix[f * n + t] : (f == t ? 1.f : 0.f)) : 0.f;
  }
  for (int i = threadIdx.x; i < SM; i += NT) {
    wo[i] = i < n ? (a.out != nullptr ? a.out[i] : 1.f) : 0.f;
    wr[i] = i < n ? (a.rd != nullptr ? a.rd[i] : 1.f) : 0.f;
  }
  pdl_wait();
  __syncthreads();
  const long long t = blockIdx.x;
  float* x = a.x + t * n * D;
  float sw = 0.f;
  for (int i = 0; i < a.same_n; ++i) sw += a.same_w[t * a.same_ld + i];
  const AT* same = reinterpret_cast<const AT*>(a.same) + t * D;
  const bf16* er = nullptr;
  if (a.tokens != nullptr) {
    int tok = a.tokens[t];
    tok = tok < 0 ? 0 : (tok >= a.V ? a.V - 1 : tok);
    er = a.emb + (long long)tok * D;
  }
  float sum = 0.f;
  for (int i = threadIdx.x * VEC; i < D; i += NT * VEC) {
    HyVec<VEC> xs[SM], u;
#pragma unroll
    for (int e = 0; e < VEC; ++e) u.v[e] = 0.f;
    if (er != nullptr) {
      HyVec<VEC> v = hy_ldv<VEC>(er + i);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] *= a.emb_scale;
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        if (s >= n) break;
        hy_stv<VEC>(x + (long long)s * D + i, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(wr[s], v.v[e], u.v[e]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < n) xs[s] = hy_ldv<VEC>(x + (long long)s * D + i);
      if (branch) {
        HyVec<VEC> y;
        if constexpr (VEC > 1) {
          if (a.y.h != nullptr) y = hy_ldv<VEC>(a.y.h + t * a.y.ld + i);
          else y = hy_ldv<VEC>(a.y.f + t * a.y.ld + i);
          if (a.y.bias != nullptr) {
            const HyVec<VEC> b = hy_ldv<VEC>(a.y.bias + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) y.v[e] += b.v[e];
          }
        } else {
          y.v[0] = lin_at(a.y, t, i);
        }
        if (sw != 0.f) {
          const HyVec<VEC> h = hy_ldv<VEC>(same + i);
#pragma unroll
          for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(sw, h.v[e], y.v[e]);
        }
#pragma unroll
        for (int j = 0; j < SM; ++j) {
          if (j >= n) break;
          HyVec<VEC> v;
#pragma unroll
          for (int e = 0; e < VEC; ++e) v.v[e] = wo[j] * y.v[e];
#pragma unroll
          for (int s = 0; s < SM; ++s) {
            if (s >= n) break;
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] = fmaf(wm[s * SM + j], xs[s].v[e], v.v[e]);
          }
          hy_stv<VEC>(x + (long long)j * D + i, v);
#pragma unroll
          for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(wr[j], v.v[e], u.v[e]);
        }
      } else {
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < n)
#pragma unroll
            for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(wr[s], xs[s].v[e], u.v[e]);
      }
    }
    hy_stv<VEC>(row + i, u);
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum += a.norm == XB_NORM_LAYER ? u.v[e] : u.v[e] * u.v[e];
  }
  if (a.hn == nullptr && a.ha == nullptr) return;
  sum = block_sum<NT>(sum, red);
  float mean = 0.f, inv;
  if (a.norm == XB_NORM_LAYER) {
    mean = sum / (float)D;
    float sq = 0.f;
    for (int i = threadIdx.x * VEC; i < D; i += NT * VEC)
#pragma unroll
      for (int e = 0; e < VEC; ++e) { const float d = row[i + e] - mean; sq = fmaf(d, d, sq); }
    inv = 1.0f / sqrtf(block_sum<NT>(sq, red) / (float)D + a.eps);
  } else {
    inv = 1.0f / sqrtf(sum / (float)D + a.eps);
  }
  for (int i = threadIdx.x * VEC; i < D; i += NT * VEC) {
    HyVec<VEC> v = hy_ldv<VEC>(row + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v.v[e] = (v.v[e] - mean) * inv * hy_norm_weight(a.nw, a.nw_mode, i + e);
    if (a.hn != nullptr) hy_stv<VEC>(a.hn + t * D + i, v);
    if (a.ha != nullptr) hy_stv<VEC>(reinterpret_cast<AT*>(a.ha) + t * D + i, v);
  }
}

// out[t] = sum of the copies (what a reader of the residual stream after a layer gets)
__global__ void hy_stream_sum_kernel(const float* __restrict__ x, float* __restrict__ out, int n, int D) {
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int i = blockIdx.y * blockDim.x + threadIdx.x;
  if (i >= D) return;
  float v = 0.f;
  for (int s = 0; s < n; ++s) v += x[(t * n + s) * D + i];
  out[t * D + i] = v;
}

// The same for steps of few rows: a row's channels are shared out over the gridDim.y blocks of a thread-block cluster (more loads in flight while
// split-K planes are summed); mean and squared deviations of the blocks' parts are merged across the cluster.
// grid (T, blocks per row), 256 threads; dynamic shared memory: ceil(D / blocks) floats.
template <typename AT, int SM>
__global__ void __launch_bounds__(256) hy_hyper_cluster_kernel(HyperArgs a) {
  namespace cg = cooperative_groups;
  extern __shared__ __align__(16) float row[];
  __shared__ float wm[SM * SM], wo[SM], wr[SM];
  __shared__ float red[32], part[2];
  const int n = a.n, D = a.D, nb = gridDim.y;
  pdl_launch_dependents();
  for (int i = threadIdx.x; i < SM * SM; i += 256) {
    const int f = i / SM, t = i - f * SM;
    wm[i] = (f < n && t < n) ? (a.mix != nullptr ? a.mix[f * n + t] : (f == t ? 1.f : 0.f)) : 0.f;
  }
  for (int i = threadIdx.x; i < SM; i += 256) {
    wo[i] = i < n ? (a.out != nullptr ? a.out[i] : 1.f) : 0.f;
    wr[i] = i < n ? (a.rd != nullptr ? a.rd[i] : 1.f) : 0.f;
  }
  pdl_wait();
  __syncthreads();
  const long long t = blockIdx.x;
  const int per = (D + nb - 1) / nb, c0 = blockIdx.y * per, nc = D - c0 < per ? (D - c0 > 0 ? D - c0 : 0) : per;
  float* x = a.x + t * n * D + c0;
  float sw = 0.f;
  for (int i = 0; i < a.same_n; ++i) sw += a.same_w[t * a.same_ld + i];
  const AT* same = reinterpret_cast<const AT*>(a.same) + t * D + c0;
  float sum = 0.f;
  for (int i = threadIdx.x; i < nc; i += 256) {
    float xs[SM], u = 0.f;
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < n) xs[s] = x[(long long)s * D + i];
    float y = lin_at(a.y, t, c0 + i);
    if (sw != 0.f) y = fmaf(sw, act_load<AT>(same + i), y);
#pragma unroll
    for (int j = 0; j < SM; ++j) {
      if (j >= n) break;
      float v = wo[j] * y;
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        if (s >= n) break;
        v = fmaf(wm[s * SM + j], xs[s], v);
      }
      x[(long long)j * D + i] = v;
      u = fmaf(wr[j], v, u);
    }
    row[i] = u;
    sum += u;
  }
  // mean and squared deviations of this block's channels, then of the row (every block merges the parts in the same order)
  float mean = a.norm == XB_NORM_LAYER ? block_sum<256>(sum, red) / (float)(nc > 0 ? nc : 1) : 0.f, sq = 0.f;
  for (int i = threadIdx.x; i < nc; i += 256) { const float d = row[i] - mean; sq = fmaf(d, d, sq); }
  sq = block_sum<256>(sq, red);
  cg::cluster_group cl = cg::this_cluster();
  if (threadIdx.x == 0) { part[0] = mean; part[1] = sq; }
  cl.sync();
  float cnt = 0.f, mu = 0.f, m2 = 0.f;
  for (int b = 0; b < nb; ++b) {
    const float* p = cl.map_shared_rank(part, b);
    const int left = D - b * per;
    const float k = (float)(left < per ? (left > 0 ? left : 0) : per);
    if (k == 0.f) continue;
    const float d = p[0] - mu, tot = cnt + k;
    m2 += p[1] + d * d * (cnt * k / tot);
    mu += d * (k / tot);
    cnt = tot;
  }
  cl.sync();   // no block leaves while its part may still be read
  const float inv = 1.0f / sqrtf(m2 / (float)D + a.eps);
  for (int i = threadIdx.x; i < nc; i += 256) {
    const float v = (row[i] - mu) * inv * hy_norm_weight(a.nw, a.nw_mode, c0 + i);
    if (a.hn != nullptr) a.hn[t * D + c0 + i] = v;
    if (a.ha != nullptr) act_store<AT>(reinterpret_cast<AT*>(a.ha) + t * D + c0 + i, v);
  }
}
