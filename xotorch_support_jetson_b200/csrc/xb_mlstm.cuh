// The matrix memory of xLSTM (XB_MIX_MLSTM) around the recurrence kernels.  Included by xb_hybrid_kernels.cuh.
//
// Per head, with log gates i = cap tanh(zi / cap), f = log sigmoid(cap tanh(zf / cap)) and a running maximum m (0 before the first token):
//   m <- max(f + m', i),   w = e^(f + m' - m),   b = e^(i - m)
//   S <- w S + (b k) v^T,  n <- w n + b k,       o = S^T q / (max(|n . q|, e^-m) + 1e-6),   q already times dim^-1/2
// The normaliser is one more value column whose value is always 1, so state and recurrence carry dvp = dv + 1 columns, rounded up to a
// multiple of four (the rest stays zero): layout [H][dvp][dk] per slot, then [H] running maxima.  Everything is fp32.
#pragma once

__host__ __device__ constexpr int hy_mlstm_cols(int dv) { return (dv + 4) & ~3; }

__device__ __forceinline__ float hy_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float hy_soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

// The scalar recurrence of one (sequence, head): w -> decay[t, h], b -> beta[t, h], e^-m -> em[t, h], the last m -> the slot.
// m_t = max(F + m_0, I) where (F, I) composes the steps up to t, (f1, i1) then (f2, i2) = (f1 + f2, max(i1 + f2, i2)): the threads compose
// stretches of the tokens, scan over the threads, then walk their stretch once more from its start.
// grid (H, n_seqs), HY_GATE_THREADS threads.
#define HY_GATE_THREADS 1024
__global__ void __launch_bounds__(HY_GATE_THREADS) hy_mlstm_gates_kernel(LinOut P, int off_i, int off_f, float cap, float* __restrict__ mstate, long long state_stride,
                                                             float* __restrict__ decay, float* __restrict__ beta, float* __restrict__ em, int H,
                                                             BatchMeta m) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sF[HY_GATE_THREADS], sI[HY_GATE_THREADS];
  const int h = blockIdx.x, tid = threadIdx.x;
  const SeqSpan sp = seq_span(m, blockIdx.y);
  float* slot_m = mstate + (long long)sp.slot * state_stride + h;
  const float m0 = sp.pos0 > 0 ? *slot_m : 0.f;
  const int per = (sp.len + HY_GATE_THREADS - 1) / HY_GATE_THREADS, t0 = tid * per, t1 = t0 + per < sp.len ? t0 + per : sp.len;
  float F = 0.f, I = -INFINITY;
  for (int t = t0; t < t1; ++t) {
    const long long r = sp.start + t;
    const float i = hy_soft_cap(lin_at(P, r, off_i + h), cap), f = hy_log_sigmoid(hy_soft_cap(lin_at(P, r, off_f + h), cap));
    beta[r * H + h] = i;
    decay[r * H + h] = f;
    I = fmaxf(I + f, i);
    F += f;
  }
  sF[tid] = F; sI[tid] = I;
  __syncthreads();
  for (int off = 1; off < HY_GATE_THREADS; off <<= 1) {   // inclusive scan of the stretches
    float pf = 0.f, pi = -INFINITY;
    if (tid >= off) { pf = sF[tid - off]; pi = sI[tid - off]; }
    __syncthreads();
    if (tid >= off) { sI[tid] = fmaxf(pi + sF[tid], sI[tid]); sF[tid] += pf; }
    __syncthreads();
  }
  float mx = tid > 0 ? fmaxf(sF[tid - 1] + m0, sI[tid - 1]) : m0;
  for (int t = t0; t < t1; ++t) {
    const long long at = (sp.start + t) * (long long)H + h;
    const float i = beta[at], f = decay[at] + mx;
    mx = fmaxf(f, i);
    decay[at] = expf(f - mx);
    beta[at] = expf(i - mx);
    em[at] = expf(-mx);
  }
  if (t0 < t1 && t1 == sp.len) *slot_m = mx;
}

// c row = [q * scale (H dk) | b k (H dk) | per head: v (dv), 1, zeros (dvp)].  VEC = 8: the projection is one bf16 matrix with 16-byte aligned
// columns, dk and dv multiples of 8; a unit is 8 channels of q, k or v, or the tail of a head's value row.
// grid (T, ceil(units / 256)), 256 threads.
template <int VEC>
__global__ void __launch_bounds__(256) hy_mlstm_prep_kernel(LinOut P, int off_q, int off_k, int off_v, float scale, const float* __restrict__ beta,
                                                            float* __restrict__ c, long long ldc, int H, int dk, int dv) {
  pdl_launch_dependents();
  pdl_wait();
  const long long t = blockIdx.x;
  const int dvp = hy_mlstm_cols(dv), HK = H * dk, nk = HK / VEC, nv = H * dv / VEC;
  const int u = blockIdx.y * 256 + threadIdx.x;
  float* row = c + t * ldc;
  if (u < 2 * nk + nv) {
    const int part = u < nk ? 0 : (u < 2 * nk ? 1 : 2), i = (u - (part == 0 ? 0 : (part == 1 ? nk : 2 * nk))) * VEC;
    const int col = (part == 0 ? off_q : (part == 1 ? off_k : off_v)) + i;
    float v[VEC];
    hy_prep_load<VEC>(P, t, col, v);
    const float f = part == 0 ? scale : (part == 1 ? beta[t * H + i / dk] : 1.0f);
    float* dst = row + (part == 0 ? i : (part == 1 ? HK + i : 2 * HK + (i / dv) * dvp + i % dv));
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= f;
    if constexpr (VEC == 8) hy_st8f(dst, v);
    else *dst = v[0];
  } else if (u < 2 * nk + nv + H) {
    float* dst = row + 2 * HK + (u - 2 * nk - nv) * dvp + dv;
    for (int e = 0; e < dvp - dv; ++e) dst[e] = e == 0 ? 1.0f : 0.0f;
  }
}

// Read-out of the recurrence o [T][H][dvp] (column dv: n . q) -> out[t, h dv + j] = out_scale * unit(o / den) * nw * sigmoid(gate), a warp per
// (token, head).  grid ceil(T * H / 8), 256 threads.
template <typename AT>
__global__ void __launch_bounds__(256) hy_mlstm_out_kernel(const float* __restrict__ o, const float* __restrict__ em, const float* __restrict__ nw, LinOut P,
                                                           int off_g, float eps, float out_scale, AT* __restrict__ out, long long ld_out, int T, int H,
                                                           int dv) {
  pdl_launch_dependents();
  pdl_wait();
  const long long th = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (th >= (long long)T * H) return;
  const long long t = th / H;
  const int h = (int)(th - t * H), dvp = hy_mlstm_cols(dv);
  const float* p = o + th * dvp;
  const float den = 1.0f / (fmaxf(fabsf(p[dv]), em[th]) + 1e-6f);
  AT* dst = out + t * ld_out + (long long)h * dv;
  float ss = 0.f;
  for (int j = lane; j < dv; j += 32) { const float v = p[j] * den; ss = fmaf(v, v, ss); }
  const float inv = out_scale / sqrtf(warp_sum(ss) / (float)dv + eps);
  for (int j = lane; j < dv; j += 32)
    act_store<AT>(dst + j, p[j] * den * inv * nw[h * dv + j] * hy_sigmoid(lin_at(P, t, off_g + h * dv + j)));
}

// The same on 32- and 16-byte accesses: eight neighbouring channels per thread, dv / 8 (a power of two up to 32) neighbouring lanes per head, gate from
// one bf16 matrix.  off_g, the pitches and dv are multiples of 8.  grid ceil(T * H * dv / 8 / 256), 256 threads.
template <typename AT>
__global__ void __launch_bounds__(256) hy_mlstm_out_vec_kernel(const float* __restrict__ o, const float* __restrict__ em, const float* __restrict__ nw,
                                                               const bf16* __restrict__ g, long long ldg, const float* __restrict__ gbias, float eps,
                                                               float out_scale, AT* __restrict__ out, long long ld_out, int T, int H, int dv) {
  pdl_launch_dependents();
  pdl_wait();
  const int per = dv >> 3, dvp = hy_mlstm_cols(dv);
  const long long idx = (long long)blockIdx.x * 256 + threadIdx.x, n = (long long)T * H * per;
  const bool live = idx < n;
  const long long th = (live ? idx : n - 1) / per;
  const int j = (int)((live ? idx : n - 1) - th * per) << 3;
  const long long t = th / H;
  const int h = (int)(th - t * H);
  float v[8], wv[8], gv[8];
  hy_ld8f(o + th * dvp + j, v);
  const float den = 1.0f / (fmaxf(fabsf(o[th * dvp + dv]), em[th]) + 1e-6f);
  hy_load8(g + t * ldg + (long long)h * dv + j, gbias != nullptr ? gbias + h * dv + j : nullptr, gv);
  hy_ld8f(nw + (long long)h * dv + j, wv);
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) { v[i] *= den; ss = fmaf(v[i], v[i], ss); }
  for (int off = per >> 1; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);   // per divides 32: lanes of a head stay together
  const float inv = out_scale / sqrtf(ss / (float)dv + eps);
#pragma unroll
  for (int i = 0; i < 8; ++i) v[i] = v[i] * inv * wv[i] * hy_sigmoid(gv[i]);
  if (live) hy_st8a<AT>(out + t * ld_out + (long long)h * dv + j, v);
}

// A step of single tokens: everything between the input and the output projection in one kernel, a block per (sequence, head).
// A warp takes one column of the state after the other, the normaliser's (value 1) among them.
// Dynamic shared memory: 2 dk (rounded up to 4) + 3 dv + 1 floats.  grid (n_seqs, H), 512 threads.
template <typename AT>
__global__ void __launch_bounds__(512) hy_mlstm_token_kernel(LinOut P, int off_q, int off_k, int off_v, int off_g, int off_i, int off_f, float cap, float scale,
                                                             float* __restrict__ state, float* __restrict__ mstate, long long state_stride,
                                                             const float* __restrict__ nw, float eps, float out_scale, AT* __restrict__ out,
                                                             long long ld_out, BatchMeta m, int H, int dk, int dv) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float gsm[];
  __shared__ float red[32], gate[3];   // fade, write strength, e^-m
  const int s = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = 16;
  const int row = m.seq_last[s], dk4 = (dk + 3) & ~3, dvp = hy_mlstm_cols(dv);
  const long long slot = m.seq_slot[s];
  const bool have = m.tok_pos[row] > 0;
  float *q = gsm, *k = q + dk4, *v = k + dk4, *g = v + dv, *o = g + dv;
  if (threadIdx.x == 511) {
    const float i = hy_soft_cap(lin_at(P, row, off_i + h), cap);
    float* sm = mstate + slot * state_stride + h;
    const float f = hy_log_sigmoid(hy_soft_cap(lin_at(P, row, off_f + h), cap)) + (have ? *sm : 0.f), mx = fmaxf(f, i);
    *sm = mx;
    gate[0] = expf(f - mx); gate[1] = expf(i - mx); gate[2] = expf(-mx);
  }
  for (int u = threadIdx.x; u < 2 * dk + 2 * dv; u += 512) {
    if (u < dk) q[u] = lin_at(P, row, off_q + h * dk + u) * scale;
    else if (u < 2 * dk) k[u - dk] = lin_at(P, row, off_k + h * dk + u - dk);
    else if (u < 2 * dk + dv) v[u - 2 * dk] = lin_at(P, row, off_v + h * dv + u - 2 * dk);
    else g[u - 2 * dk - dv] = lin_at(P, row, off_g + h * dv + u - 2 * dk - dv);
  }
  __syncthreads();
  const float w = gate[0], b = gate[1];
  float* st = state + slot * state_stride + (long long)h * dvp * dk;
  const bool al = (dk & 3) == 0 && (reinterpret_cast<uintptr_t>(st) & 15) == 0;
#pragma unroll 4
  for (int j = warp; j <= dv; j += nwarps) {
    float* col = st + (long long)j * dk;
    const float vj = j < dv ? v[j] * b : b;
    float acc = 0.f;
    if (al) {
      for (int i = lane * 4; i < dk; i += 128) {
        float4 S = have ? *reinterpret_cast<const float4*>(col + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 k4 = *reinterpret_cast<const float4*>(k + i), q4 = *reinterpret_cast<const float4*>(q + i);
        S.x = fmaf(w, S.x, k4.x * vj); S.y = fmaf(w, S.y, k4.y * vj); S.z = fmaf(w, S.z, k4.z * vj); S.w = fmaf(w, S.w, k4.w * vj);
        *reinterpret_cast<float4*>(col + i) = S;
        acc = fmaf(q4.x, S.x, acc); acc = fmaf(q4.y, S.y, acc); acc = fmaf(q4.z, S.z, acc); acc = fmaf(q4.w, S.w, acc);
      }
    } else {
      for (int i = lane; i < dk; i += 32) {
        const float S = fmaf(w, have ? col[i] : 0.f, k[i] * vj);
        col[i] = S;
        acc = fmaf(q[i], S, acc);
      }
    }
    acc = warp_sum(acc);
    if (lane == 0) o[j] = acc;
  }
  __syncthreads();
  const float den = 1.0f / (fmaxf(fabsf(o[dv]), gate[2]) + 1e-6f);
  float ss = 0.f;
  for (int j = threadIdx.x; j < dv; j += 512) ss = fmaf(o[j] * den, o[j] * den, ss);
  const float inv = out_scale / sqrtf(block_sum<512>(ss, red) / (float)dv + eps);
  for (int j = threadIdx.x; j < dv; j += 512)
    act_store<AT>(out + (long long)row * ld_out + (long long)h * dv + j, o[j] * den * inv * nw[h * dv + j] * hy_sigmoid(g[j]));
}
