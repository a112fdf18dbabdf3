// From the projected q | k | v of a token row to what softmax attention reads: short causal filter, whole-projection norms, query
// temperature, rotation, unit heads, cache append -- each switched by its field.  Included by xb_hybrid_kernels.cuh.
#pragma once
#include <cooperative_groups.h>

// Columns [off_q, off_q + H dk + G dk + G dv) of the projection are q | k | v, channel c of the filter is column off_q + c.
// kp / vp: entries of a query / key row and of a value row in the pools and in qg, >= dk / dv (tensor-core kernels read whole
// 64- or 128-wide rows; what lies behind dk / dv is zero: queries are written with their zeros, pools keep those they were cleared to).
struct QkvPrep {
  int off_q, H, G, dk, dv, kp, vp;
  int taps;                 // 0 = no filter; weights [channels][taps], the slot's tail [taps - 1][channels] (oldest first)
  const float* conv_w;
  float* tail;
  long long tail_stride;
  int write_tail;           // a step of single tokens: the kernel also moves the tail on (hy_qkv_prep_kernel)
  const float *qn, *kn;     // whole-projection RMS norm weights, or nullptr
  float eps;
  float temp_coef;
  int temp_every;
  RotArgs rot;
  int head_norm;            // after the rotation: every query / key head divided by its root mean square
  float* qa;                // fp32 queries [T][H * dk], or nullptr
  bf16* qg;                 // bf16 queries [T][H * kp], or nullptr
};

// eight neighbouring channels / one channel of the projection, bias added
template <int VEC> __device__ __forceinline__ void hy_prep_load(const LinOut& P, long long row, int col, float* v) {
  if constexpr (VEC == 8) hy_load8(P.h + row * P.ld + col, P.bias != nullptr ? P.bias + col : nullptr, v);
  else v[0] = lin_at(P, row, col);
}
// channel c of a row after the filter.  start / pos0: first row of the row's sequence in this step and its position.
__device__ __forceinline__ float hy_prep_channel(const QkvPrep& a, const LinOut& P, int row, int start, int pos, int pos0, float* tl, int C, int c) {
  const float u = lin_at(P, row, a.off_q + c);
  if (a.taps == 0) return u;
  const float* w = a.conv_w + (long long)c * a.taps;
  float y = 0.f;
  for (int j = 0; j < a.taps - 1; ++j) {   // oldest first
    const int d = a.taps - 1 - j, p = pos - d;
    if (p < 0) continue;
    y = fmaf(w[j], row - d >= start ? lin_at(P, row - d, a.off_q + c) : tl[(long long)(p - (pos0 - (a.taps - 1))) * C + c], y);
  }
  y = fmaf(w[a.taps - 1], u, y);
  if (a.write_tail && a.taps > 1) {   // the row is its sequence's only one: this thread alone reads and moves this channel
    for (int j = 0; j + 2 < a.taps; ++j) tl[(long long)j * C + c] = tl[(long long)(j + 1) * C + c];
    tl[(long long)(a.taps - 2) * C + c] = u;
  }
  return y;
}

// Any sizes, any form of the projection.  A token row's heads (queries, then keys) and value heads are shared out over the gridDim.y blocks of a
// thread-block cluster, head after head; only the sums of the whole-projection norms cross them.
// grid (T, blocks per row), NT threads; dynamic shared memory ceil((H + G) / blocks) * (dk + 1) + rot.dims floats.
template <typename KT, int NT>
__global__ void __launch_bounds__(NT) hy_qkv_prep_kernel(LinOut P, QkvPrep a, KT* __restrict__ k_pool, KT* __restrict__ v_pool, BatchMeta m) {
  namespace cg = cooperative_groups;
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float qk[];
  __shared__ float red[32], part[2];
  const int row = blockIdx.x, rank = blockIdx.y, nb = gridDim.y;
  const int H = a.H, G = a.G, dk = a.dk, dv = a.dv, nq = H * dk, nk = G * dk, C = nq + nk + G * dv;
  const int heads = (H + G - rank + nb - 1) / nb, vheads = (G - rank + nb - 1) / nb;   // local head x is head rank + x * nb
  float* hinv = qk + (H + G + nb - 1) / nb * dk;
  float* cs = hinv + (H + G + nb - 1) / nb;
  const int s = m.tok_seq[row], pos = m.tok_pos[row], slot = m.seq_slot[s];
  const int start = s > 0 ? m.seq_last[s - 1] + 1 : 0, pos0 = a.taps > 1 ? m.tok_pos[start] : pos;
  float* tl = a.tail != nullptr ? a.tail + (long long)slot * a.tail_stride : nullptr;
  const long long pg = m.page_table[(long long)slot * m.max_pages + pos / m.page_tokens];
  const int ip = pos % m.page_tokens;
  const int hp = a.rot.dims >> 1;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < heads * dk + vheads * dv; i += NT) {
    if (i < heads * dk) {
      const int hd = rank + (i / dk) * nb;
      const float y = hy_prep_channel(a, P, row, start, pos, pos0, tl, C, hd * dk + i % dk);
      qk[i] = y;
      if (hd < H) sq = fmaf(y, y, sq); else sk = fmaf(y, y, sk);
    } else {
      const int iv = i - heads * dk, g = rank + (iv / dv) * nb, c = iv % dv;
      act_store<KT>(v_pool + ((pg * G + g) * m.page_tokens + ip) * a.vp + c, hy_prep_channel(a, P, row, start, pos, pos0, tl, C, nq + nk + g * dv + c));
    }
  }
  for (int j = threadIdx.x; j < hp; j += NT) hy_rot_cs(a.rot, pos, j, &cs[2 * j], &cs[2 * j + 1]);
  const float temp = a.temp_every > 0 ? 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every) + 1.0f) : 1.0f;
  float qs = temp, ks = 1.f;
  if (a.qn != nullptr) {
    sq = block_sum<NT>(sq, red);
    sk = block_sum<NT>(sk, red);
    if (nb > 1) {   // every block adds the parts in the same order
      cg::cluster_group cl = cg::this_cluster();
      if (threadIdx.x == 0) { part[0] = sq; part[1] = sk; }
      cl.sync();
      sq = sk = 0.f;
      for (int b = 0; b < nb; ++b) {
        const float* p = cl.map_shared_rank(part, b);
        sq += p[0];
        sk += p[1];
      }
      cl.sync();   // no block leaves while its sums may still be read
    }
    qs = temp / sqrtf(sq / (float)nq + a.eps);
    ks = 1.0f / sqrtf(sk / (float)nk + a.eps);
  }
  __syncthreads();
  // norm and rotation in place: a thread owns a turning pair or one entry that does not turn
  const int per = dk - hp;
  if (a.qn != nullptr || hp > 0 || a.temp_every > 0) {
    for (int u = threadIdx.x; u < heads * per; u += NT) {
      const int x = u / per, j = u - x * per, hd = rank + x * nb, base = x * dk;
      const float sc = hd < H ? qs : ks;
      const float* w = a.qn != nullptr ? (hd < H ? a.qn + hd * dk : a.kn + (hd - H) * dk) : nullptr;
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
    for (int x = warp; x < heads; x += NT / 32) {
      float ss = 0.f;
      for (int d = lane; d < dk; d += 32) ss = fmaf(qk[x * dk + d], qk[x * dk + d], ss);
      ss = warp_sum(ss);
      if (lane == 0) hinv[x] = 1.0f / sqrtf(ss / (float)dk + a.eps);
    }
    __syncthreads();
  }
  for (int i = threadIdx.x; i < heads * a.kp; i += NT) {
    const int x = i / a.kp, d = i - x * a.kp, hd = rank + x * nb;
    const float y = d < dk ? qk[x * dk + d] * (a.head_norm ? hinv[x] : 1.f) : 0.f;
    if (hd >= H) {
      if (d < dk) act_store<KT>(k_pool + ((pg * G + hd - H) * m.page_tokens + ip) * a.kp + d, y);
    } else {
      if (a.qa != nullptr && d < dk) a.qa[(long long)row * nq + hd * dk + d] = y;
      if (a.qg != nullptr) a.qg[(long long)row * H * a.kp + hd * a.kp + d] = f2bf(y);
    }
  }
}

// Prompts whose projection came back as ONE bf16 matrix, bf16 pools: a block takes RT token rows, so that a filter's weights and the rows
// it looks back to are read once for all of them; unit heads without whole-projection norms and temperature; 16-byte accesses (dk, dv, kp, vp, off_q and the pitch are multiples of 8).  TAPS: 0 = no filter.
// grid (ceil(T / RT)), 256 threads; dynamic shared memory RT * ((H + G) (dk + 1) + rot.dims) floats.
template <int TAPS, int RT>
__global__ void __launch_bounds__(256, TAPS > 0 ? 2 : 4) hy_qkv_prep_tile_kernel(LinOut P, QkvPrep a, bf16* __restrict__ k_pool, bf16* __restrict__ v_pool, BatchMeta m, int T) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int BACK = TAPS > 1 ? TAPS - 1 : 0;
  extern __shared__ __align__(16) float qk[];   // [RT][(H + G) dk], then 1 / rms per head, then cos / sin
  __shared__ float sums[8][2 * RT], scale[2 * RT];
  __shared__ long long page[RT];
  __shared__ int where[RT][5];                  // position, offset in the page, first row of its sequence, that row's position, slot
  const int r0 = blockIdx.x * RT, nr = T - r0 < RT ? T - r0 : RT;
  const int H = a.H, G = a.G, dk = a.dk, dv = a.dv, nq = H * dk, nqk = nq + G * dk, C = nqk + G * dv, NH = H + G;
  float* hinv = qk + RT * nqk;
  float* cs = hinv + RT * NH;
  const int hp = a.rot.dims >> 1, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x < RT) {
    const int row = r0 + (threadIdx.x < nr ? threadIdx.x : 0), s = m.tok_seq[row], pos = m.tok_pos[row], slot = m.seq_slot[s], start = s > 0 ? m.seq_last[s - 1] + 1 : 0;
    page[threadIdx.x] = m.page_table[(long long)slot * m.max_pages + pos / m.page_tokens];
    int* w = where[threadIdx.x];
    w[0] = pos; w[1] = pos % m.page_tokens; w[2] = start; w[3] = m.tok_pos[start]; w[4] = slot;
  }
  __syncthreads();
  for (int j = threadIdx.x; j < RT * hp; j += 256) {
    const int r = j / hp, x = j - r * hp;
    hy_rot_cs(a.rot, where[r][0], x, &cs[2 * j], &cs[2 * j + 1]);
  }
  float sq[RT], sk[RT];
#pragma unroll
  for (int r = 0; r < RT; ++r) sq[r] = sk[r] = 0.f;
  // the tile lies in one sequence: what its rows look back to is one run of rows and, in front of the step, of the slot's tail
  const bool one = where[0][2] == where[nr - 1][2];
  const int pos0 = where[0][0], start0 = where[0][2], first0 = where[0][3];
  const float* tail0 = TAPS > 1 ? a.tail + (long long)where[0][4] * a.tail_stride : nullptr;
  if (TAPS > 0 && !one) {   // rows of several sequences: each looks back by itself
#pragma unroll
    for (int r = 0; r < RT; ++r) {
      if (r >= nr) break;
      for (int c = threadIdx.x; c < C; c += 256) {
        const float y = hy_prep_channel(a, P, r0 + r, where[r][2], where[r][0], where[r][3], a.tail + (long long)where[r][4] * a.tail_stride, C, c);
        if (c < nqk) {
          if (c < nq) sq[r] = fmaf(y, y, sq[r]); else sk[r] = fmaf(y, y, sk[r]);
          qk[r * nqk + c] = y;
        } else {
          const int iv = c - nqk, g = iv / dv, d = iv - g * dv;
          v_pool[((page[r] * G + g) * m.page_tokens + where[r][1]) * a.vp + d] = f2bf(y);
        }
      }
    }
  }
  for (int c = threadIdx.x * 4; c < ((TAPS == 0 || one) ? C : 0); c += 256 * 4) {   // four channels per thread keep a filter's window in few registers
    HyVec<4> z[RT + BACK], b;
    float w[TAPS > 0 ? TAPS : 1][4];
#pragma unroll
    for (int e = 0; e < 4; ++e) b.v[e] = 0.f;
    if (P.bias != nullptr) b = hy_ldv<4>(P.bias + a.off_q + c);
#pragma unroll
    for (int i = 0; i < RT + BACK; ++i) {
      const int row = r0 - BACK + i;
      if (i >= BACK ? row < r0 + nr : row >= start0) {
        z[i] = hy_ldv<4>(P.h + (long long)row * P.ld + a.off_q + c);
#pragma unroll
        for (int e = 0; e < 4; ++e) z[i].v[e] += b.v[e];
      } else if (i < BACK && pos0 - (BACK - i) >= 0) {   // in front of this step's rows: the slot's tail
        const float* tl = tail0 + (long long)(pos0 - (BACK - i) - (first0 - BACK)) * C + c;   // (a slot's state has no alignment of its own)
#pragma unroll
        for (int e = 0; e < 4; ++e) z[i].v[e] = tl[e];
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) z[i].v[e] = 0.f;
      }
    }
    if (TAPS > 0) {
#pragma unroll
      for (int x = 0; x < (TAPS > 0 ? TAPS : 1); ++x) {   // four channels' taps are 4 TAPS neighbouring numbers
        const HyVec<4> t = hy_ldv<4>(a.conv_w + (long long)c * TAPS + 4 * x);
#pragma unroll
        for (int e = 0; e < 4; ++e) w[(4 * x + e) % (TAPS > 0 ? TAPS : 1)][(4 * x + e) / (TAPS > 0 ? TAPS : 1)] = t.v[e];
      }
    }
#pragma unroll
    for (int r = 0; r < RT; ++r) {
      if (r >= nr) break;
      HyVec<4> y;
      if (TAPS == 0) {
        y = z[r + BACK];
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          y.v[e] = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) y.v[e] = fmaf(w[j][e], z[r + j].v[e], y.v[e]);   // oldest first
        }
      }
      if (c < nqk) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) ss = fmaf(y.v[e], y.v[e], ss);
        if (c < nq) sq[r] += ss; else sk[r] += ss;
        hy_stv<4>(qk + r * nqk + c, y);
      } else {
        const int iv = c - nqk, g = iv / dv, d = iv - g * dv;
        hy_stv<4>(v_pool + ((page[r] * G + g) * m.page_tokens + where[r][1]) * a.vp + d, y);
      }
    }
  }
  if (a.qn != nullptr) {
#pragma unroll
    for (int r = 0; r < RT; ++r) {
      const float x = warp_sum(sq[r]), y = warp_sum(sk[r]);
      if (lane == 0) { sums[warp][r] = x; sums[warp][RT + r] = y; }
    }
  }
  __syncthreads();
  if (threadIdx.x < 2 * RT) {
    const int r = threadIdx.x % RT;
    const bool q = threadIdx.x < RT;
    float v = 1.f;
    if (a.qn != nullptr) {
      float s = 0.f;
#pragma unroll
      for (int x = 0; x < 8; ++x) s += sums[x][threadIdx.x];
      v = 1.0f / sqrtf(s / (float)(q ? nq : nqk - nq) + a.eps);
    }
    if (q && a.temp_every > 0) v *= 1.0f + a.temp_coef * logf((float)((where[r][0] + 1) / a.temp_every) + 1.0f);
    scale[threadIdx.x] = v;
  }
  if (a.head_norm) {   // the rotation multiplies a pair's length by rot.mult and nothing else, so the sums can be taken in front of it
    const float m2 = a.rot.mult * a.rot.mult;
    const int l8 = lane & 7;
    for (int x = threadIdx.x >> 3; x < nr * NH; x += 32) {   // eight lanes per head; a whole warp leaves or stays with its eighth
      const float* p = qk + (x / NH) * nqk + (x % NH) * dk;
      float ss = 0.f;
      for (int d = l8 * 4; d < dk; d += 32) {
        const float4 v = *reinterpret_cast<const float4*>(p + d);
        const float f[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) ss = fmaf(f[e] * f[e], d + e < a.rot.dims ? m2 : 1.f, ss);
      }
      const unsigned mask = 0xffu << (lane & 24);
#pragma unroll
      for (int off = 1; off < 8; off <<= 1) ss += __shfl_xor_sync(mask, ss, off);
      if (l8 == 0) hinv[x] = 1.0f / sqrtf(ss / (float)dk + a.eps);
    }
  }
  __syncthreads();
  const int dk8 = dk >> 3, hv = hp & ~7;   // hv: half-split partners lie a multiple of eight entries away when hp is one
  for (int u = threadIdx.x; u < nr * NH * dk8; u += 256) {
    const int r = u / (NH * dk8), rem = u - r * NH * dk8, hd = rem / dk8, d = (rem - hd * dk8) << 3;
    const float* p = qk + r * nqk + hd * dk;
    const float* ct = cs + 2 * hp * r;
    const bool is_q = hd < H;
    const float sc = scale[is_q ? r : RT + r];
    const float* nw = a.qn != nullptr ? (is_q ? a.qn + hd * dk : a.kn + (hd - H) * dk) : nullptr;
    float x[8], y[8];
    hy_ld8f(p + d, x);
    if (nw != nullptr) {
      float w[8];
      hy_ld8f(nw + d, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] *= sc * w[e];
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] *= sc;
    }
    if (d >= a.rot.dims) {
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] = x[e];
    } else if (!a.rot.half) {
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        const bool turns = d + e < a.rot.dims;
        const float c = turns ? ct[d + e] : 1.f, sn = turns ? ct[d + e + 1] : 0.f;
        y[e] = x[e] * c - x[e + 1] * sn;
        y[e + 1] = x[e + 1] * c + x[e] * sn;
      }
    } else {
      float z[8];   // the partners
      if (hv == hp) {
        const int dp = d < hp ? d + hp : d - hp;
        hy_ld8f(p + dp, z);
        if (nw != nullptr) {
          float w[8];
          hy_ld8f(nw + dp, w);
#pragma unroll
          for (int e = 0; e < 8; ++e) z[e] *= sc * w[e];
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) z[e] *= sc;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int dp = d + e < hp ? d + e + hp : d + e - hp;
          z[e] = d + e < a.rot.dims ? p[dp] * sc * (nw != nullptr ? nw[dp] : 1.f) : 0.f;
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const bool turns = d + e < a.rot.dims, first = d + e < hp;
        const int j = first ? d + e : d + e - hp;
        const float c = turns ? ct[2 * j] : 1.f, sn = turns ? ct[2 * j + 1] : 0.f;
        y[e] = first ? x[e] * c - z[e] * sn : x[e] * c + z[e] * sn;
      }
    }
    if (a.head_norm) {
      const float f = hinv[r * NH + hd];
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] *= f;
    }
    bf16* dst = is_q ? a.qg + (long long)(r0 + r) * H * a.kp + hd * a.kp + d : k_pool + ((page[r] * G + hd - H) * m.page_tokens + where[r][1]) * a.kp + d;
    *reinterpret_cast<uint4*>(dst) = hy_pack8(y);
  }
  if (a.kp > dk) {   // the queries' padding
    const int z8 = (a.kp - dk) >> 3;
    for (int u = threadIdx.x; u < nr * H * z8; u += 256) {
      const int r = u / (H * z8), rem = u - r * H * z8, h = rem / z8;
      *reinterpret_cast<uint4*>(a.qg + (long long)(r0 + r) * H * a.kp + h * a.kp + dk + ((rem - h * z8) << 3)) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
}
