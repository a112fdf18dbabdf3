// From the projected q | k | v of a token row to what softmax attention reads: short causal filter, whole-projection norms, query
// temperature, rotation, unit heads, cache append -- each switched by its field.  Included by xb_hybrid_kernels.cuh.
#pragma once

// Columns [off_q, off_q + H dk + G dk + G dv) of the projection are q | k | v, channel c of the filter is column off_q + c.
// kp / vp: entries of a query / key row and of a value row in the pools and in qg, >= dk / dv (tensor-core kernels read whole
// 64- or 128-wide rows; what lies behind dk / dv is zero: queries are written with their zeros, pools keep those they were cleared to).
struct QkvPrep {
  int off_q, H, G, dk, dv, kp, vp;
  int taps;                 // 0 = no filter; weights [channels][taps], the slot's tail [taps - 1][channels] (oldest first)
  const float* conv_w;
  float* tail;
  long long tail_stride;
  int write_tail;           // a step of single tokens: the kernel also moves the tail on
  const float *qn, *kn;     // whole-projection RMS norm weights, or nullptr
  float eps;
  float temp_coef;
  int temp_every;
  RotArgs rot;
  int head_norm;            // after the rotation: every query / key head divided by its root mean square
  float* qa;                // fp32 queries [T][H * dk], or nullptr
  bf16* qg;                 // bf16 queries [T][H * kp], or nullptr
};

// VEC neighbouring channels of the projection (bias added), VEC = 8 on a bf16 matrix with 16-byte aligned rows
template <int VEC> __device__ __forceinline__ void hy_prep_load(const LinOut& P, long long row, int col, float* v) {
  if constexpr (VEC == 8) hy_load8(P.h + row * P.ld + col, P.bias != nullptr ? P.bias + col : nullptr, v);
  else v[0] = lin_at(P, row, col);
}
// channels c .. c + VEC - 1 of a row after the filter.  start / pos0: first row of the row's sequence in this step and its position.
template <int VEC>
__device__ __forceinline__ void hy_prep_channels(const QkvPrep& a, const LinOut& P, int row, int start, int pos, int pos0, float* tl, int C, int c, float* y) {
  float u[VEC];
  hy_prep_load<VEC>(P, row, a.off_q + c, u);
  if (a.taps == 0) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = u[e];
    return;
  }
  const float* w = a.conv_w + (long long)c * a.taps;
#pragma unroll
  for (int e = 0; e < VEC; ++e) y[e] = 0.f;
  for (int j = 0; j < a.taps - 1; ++j) {   // oldest first
    const int d = a.taps - 1 - j, p = pos - d;
    if (p < 0) continue;
    float z[VEC];
    if (row - d >= start) {
      hy_prep_load<VEC>(P, row - d, a.off_q + c, z);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) z[e] = tl[(long long)(p - (pos0 - (a.taps - 1))) * C + c + e];
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = fmaf(w[e * a.taps + j], z[e], y[e]);
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) y[e] = fmaf(w[e * a.taps + a.taps - 1], u[e], y[e]);
  if (a.write_tail) {   // the row is its sequence's only one: this thread alone reads and moves these channels
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      for (int j = 0; j + 2 < a.taps; ++j) tl[(long long)j * C + c + e] = tl[(long long)(j + 1) * C + c + e];
      if (a.taps > 1) tl[(long long)(a.taps - 2) * C + c + e] = u[e];
    }
  }
}

// grid (T), NT threads; dynamic shared memory ((H + G) dk + (H + G) + rot.dims) floats.  VEC = 8 wants bf16 pools, dk, dv, kp, vp, off_q
// multiples of 8 and the projection as one bf16 matrix with a pitch that is one too.
template <typename KT, int NT, int VEC>
__global__ void __launch_bounds__(NT) hy_qkv_prep_kernel(LinOut P, QkvPrep a, KT* __restrict__ k_pool, KT* __restrict__ v_pool, BatchMeta m) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float qk[];
  __shared__ float red[32];
  const int row = blockIdx.x;
  const int H = a.H, G = a.G, dk = a.dk, dv = a.dv, nq = H * dk, nk = G * dk, nv = G * dv, C = nq + nk + nv;
  float* hinv = qk + nq + nk;
  float* cs = hinv + H + G;
  const int s = m.tok_seq[row], pos = m.tok_pos[row], slot = m.seq_slot[s];
  const int start = s > 0 ? m.seq_last[s - 1] + 1 : 0, pos0 = a.taps > 1 ? m.tok_pos[start] : pos;
  float* tl = a.tail != nullptr ? a.tail + (long long)slot * a.tail_stride : nullptr;
  const long long pg = m.page_table[(long long)slot * m.max_pages + pos / m.page_tokens];
  const int ip = pos % m.page_tokens;
  const int hp = a.rot.dims >> 1;
  for (int j = threadIdx.x; j < hp; j += NT) hy_rot_cs(a.rot, pos, j, &cs[2 * j], &cs[2 * j + 1]);
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x * VEC; i < C; i += NT * VEC) {
    float y[VEC];
    hy_prep_channels<VEC>(a, P, row, start, pos, pos0, tl, C, i, y);
    if (i < nq + nk) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) { qk[i + e] = y[e]; ss = fmaf(y[e], y[e], ss); }
      if (i < nq) sq += ss; else sk += ss;
    } else {
      const int iv = i - nq - nk, g = iv / dv, c = iv - g * dv;
      KT* dst = v_pool + ((pg * G + g) * m.page_tokens + ip) * a.vp + c;
      if constexpr (VEC == 8) *reinterpret_cast<uint4*>(dst) = hy_pack8(y);
      else act_store<KT>(dst, y[0]);
    }
  }
  const float temp = a.temp_every > 0 ? 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every) + 1.0f) : 1.0f;
  float qs = temp, ks = 1.f;
  if (a.qn != nullptr) {
    qs = temp / sqrtf(block_sum<NT>(sq, red) / (float)nq + a.eps);
    ks = 1.0f / sqrtf(block_sum<NT>(sk, red) / (float)nk + a.eps);
  }
  __syncthreads();
  // norm and rotation in place: a thread owns a turning pair or one entry that does not turn
  const int per = dk - hp;
  if (a.qn != nullptr || hp > 0 || a.temp_every > 0) {
    for (int u = threadIdx.x; u < (H + G) * per; u += NT) {
      const int hd = u / per, j = u - hd * per, base = hd * dk;
      const float sc = hd < H ? qs : ks;
      const float* w = a.qn != nullptr ? (hd < H ? a.qn + base : a.kn + (base - nq)) : nullptr;
      if (j < hp) {
        const int d0 = a.rot.half ? j : 2 * j, d1 = a.rot.half ? j + hp : 2 * j + 1;
        float x0 = qk[base + d0] * sc, x1 = qk[base + d1] * sc;
        if (w != nullptr) { x0 *= w[d0]; x1 *= w[d1]; }
        const float c = cs[2 * j], sn = cs[2 * j + 1];
        qk[base + d0] = x0 * c - x1 * sn;
        qk[base + d1] = x1 * c + x0 * sn;
      } else {
        const int d = a.rot.dims + (j - hp);
        qk[base + d] *= w != nullptr ? sc * w[d] : sc;
      }
    }
    __syncthreads();
  }
  if (a.head_norm) {   // a warp per head
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int hd = warp; hd < H + G; hd += NT / 32) {
      float ss = 0.f;
      for (int d = lane; d < dk; d += 32) ss = fmaf(qk[hd * dk + d], qk[hd * dk + d], ss);
      ss = warp_sum(ss);
      if (lane == 0) hinv[hd] = 1.0f / sqrtf(ss / (float)dk + a.eps);
    }
    __syncthreads();
  }
  if (a.qa != nullptr)
    for (int i = threadIdx.x; i < nq; i += NT) a.qa[(long long)row * nq + i] = a.head_norm ? qk[i] * hinv[i / dk] : qk[i];
  if (a.qg != nullptr) {
    for (int i = threadIdx.x * VEC; i < H * a.kp; i += NT * VEC) {
      const int h = i / a.kp, d = i - h * a.kp;
      const float f = a.head_norm ? hinv[h] : 1.f;
      float y[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = d + e < dk ? qk[h * dk + d + e] * f : 0.f;
      bf16* dst = a.qg + (long long)row * H * a.kp + i;
      if constexpr (VEC == 8) *reinterpret_cast<uint4*>(dst) = hy_pack8(y);
      else *dst = f2bf(y[0]);
    }
  }
  for (int i = threadIdx.x * VEC; i < nk; i += NT * VEC) {
    const int g = i / dk, d = i - g * dk;
    const float f = a.head_norm ? hinv[H + g] : 1.f;
    float y[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = qk[nq + i + e] * f;
    KT* dst = k_pool + ((pg * G + g) * m.page_tokens + ip) * a.kp + d;
    if constexpr (VEC == 8) *reinterpret_cast<uint4*>(dst) = hy_pack8(y);
    else act_store<KT>(dst, y[0]);
  }
}
