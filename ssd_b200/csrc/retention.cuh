// retention.cuh — linear attention with a fixed decay per head, for the layered (hybrid) models:
//     S_t = a S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   y_t = unit_rms(o_t) * silu(g_t)        (per head; S [D, V] fp32)
// with q and k rotated (half-apart pairs, fp32 angles) and k scaled.  The decay does not depend on the data, so a portion runs in chunks
// of 64 rows that do not wait for one another: with S_c the state before chunk c, n its rows and i, j rows inside it,
//     o_i = a^(i+1) S_c^T q_i + sum_{j<=i} a^(i-j) (q_i . k_j) v_j,     S_(c+1) = a^n S_c + sum_j a^(n-1-j) k_j v_j^T.
// Only products of decays are formed, never quotients; the powers come from a table made in double.
//
//   retention_prep_kernel          rotated q and k of the rows that portions bring (fp32)
//   retention_chunk_state_*        a chunk's own sum  sum_j a^(n-1-j) k_j v_j^T, all chunks at once
//   retention_state_scan_kernel    the walk over a sequence's chunks, elementwise: every chunk's sum becomes the state before it,
//                                  the last state goes to the sequence's slot
//   retention_chunk_out_*          a chunk's rows: what the state gives plus what the chunk gives
//   retention_decode_kernel        single-token rows: rotation, one pass over the state, norm and gate in one launch
// Two forms of the chunk kernels: _mma (bf16 storage, D and V up to 128) runs on the tensor cores with every fp32 operand split into two
// bf16 terms (three products, fp32 accumulation: about 2^-16 relative) and leaves normed, gated rows; _any (any size; fp32 storage) is
// plain fp32 FMA and leaves o for head_rmsnorm_gate_kernel.  The state itself is fp32 in both.
// A slot's content is read only when the sequence has run tokens before (pos0 > 0): a reused slot needs no clearing.
#pragma once
#include "gqa_attention.cuh"  // head_row, row_angles
#include "layer_ops.cuh"

namespace ssdk {

constexpr int kRetChunk = 64;

struct RetentionArgs {
  const float* z; int ldz;    // [M, ldz]: q [H D] | k [H D] | v [H V] | g [H V] (fp32 projections)
  float* qk;                  // [M, 2 H D] rotated q | rotated, scaled k
  const float* pw;            // [H, kRetChunk + 1] decay^0 .. decay^64
  float* chunks;              // [chunk records, H, D, V]
  float* S; size_t slot_stride;
  const float* inv_freq; int rot_dims;
  void* y;                    // [M, H V] T
  float* o;                   // [M, H V] fp32 read-out before norm and gate, or nullptr (kernels that norm and gate themselves)
  int H, D, V;
  float k_scale, eps;
  int vec;                    // 1: D, V, rot_dims / 2, strides and pointers are whole groups of four floats
};

// record of chunk 0 of sequence s: sequences never overlap (a sequence with n rows has ceil(n / 64) chunks)
SSDK_DEVINL int ret_record(const Ragged& rg, int s) { return rg.cu[s] / kRetChunk + s; }

// grid (M, y): the warps of a row's CTAs take its 2 H heads in turn.  dynamic shared memory: rot_dims floats
template <int VEC>
__global__ void retention_prep_kernel(const RetentionArgs p, const Ragged rg) {
  SSDK_DYN_SMEM(float, rp_cs);
  const int m = blockIdx.x, s = rg.tok_seq[m], pos = rg.pos0[s] + (m - rg.cu[s]), half = (p.inv_freq ? p.rot_dims : 0) >> 1;
  if (rg.cu[s + 1] - rg.cu[s] == 1) return;   // (retention_decode_kernel turns its own row)
  row_angles(rp_cs, half, pos, p.inv_freq, 1.f);
  __syncthreads();
  const int nw = blockDim.x >> 5;
  for (int u = blockIdx.y * nw + (threadIdx.x >> 5); u < 2 * p.H; u += gridDim.y * nw)
    head_row<float, float, VEC>(p.z + (size_t)m * p.ldz + (size_t)u * p.D, p.qk + (size_t)m * 2 * p.H * p.D + (size_t)u * p.D, p.D, half, rp_cs,
                                (const float*)nullptr, 1.f, u < p.H ? 1.f : p.k_scale, threadIdx.x & 31);
}

// ------------------------------------------------------------------------------------------------ fp32 FMA form
// 16 x 64 slices of two operands in shared memory, 64 x 64 results, 4 x 4 per thread
struct RetTile {
  float a[16][68], b[16][68];
};
SSDK_DEVINL void ret_fma(const RetTile& t, int tx, int ty, float (&acc)[4][4]) {
#pragma unroll
  for (int kk = 0; kk < 16; ++kk) {
    const float4 a = *reinterpret_cast<const float4*>(&t.a[kk][ty * 4]), b = *reinterpret_cast<const float4*>(&t.b[kk][tx * 4]);
    const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
  }
}

// grid (chunks of the longest portion, H * ceil(D / 64) * ceil(V / 64), n_seqs), 256 threads
__global__ void __launch_bounds__(256) retention_chunk_state_any_kernel(const RetentionArgs p, const Ragged rg) {
  __shared__ __align__(16) RetTile t;
  const int s = blockIdx.z, c = blockIdx.x, r0 = rg.cu[s] + c * kRetChunk, left = rg.cu[s + 1] - r0;
  if (rg.cu[s + 1] - rg.cu[s] < 2 || left <= 0) return;
  const int n = min(left, kRetChunk), nv = (p.V + 63) / 64, nd = (p.D + 63) / 64, hd = blockIdx.y / (nd * nv), tile = blockIdx.y % (nd * nv);
  const int d0 = tile / nv * 64, v0 = tile % nv * 64, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, H = p.H, D = p.D, V = p.V;
  const float* pw = p.pw + (size_t)hd * (kRetChunk + 1);
  const float* k = p.qk + (size_t)r0 * 2 * H * D + (size_t)(H + hd) * D;
  const float* v = p.z + (size_t)r0 * p.ldz + 2 * (size_t)H * D + (size_t)hd * V;
  float acc[4][4] = {};
  for (int j0 = 0; j0 < n; j0 += 16) {
    for (int e = tid; e < 16 * 64; e += 256) {
      const int j = j0 + (e >> 6), c2 = e & 63;
      t.a[e >> 6][c2] = (j < n && d0 + c2 < D) ? k[(size_t)j * 2 * H * D + d0 + c2] * pw[n - 1 - j] : 0.f;
      t.b[e >> 6][c2] = (j < n && v0 + c2 < V) ? v[(size_t)j * p.ldz + v0 + c2] : 0.f;
    }
    __syncthreads();
    ret_fma(t, tx, ty, acc);
    __syncthreads();
  }
  float* out = p.chunks + ((size_t)(ret_record(rg, s) + c) * H + hd) * D * V;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = d0 + ty * 4 + i, vv = v0 + tx * 4 + j;
      if (d < D && vv < V) out[(size_t)d * V + vv] = acc[i][j];
    }
}

// grid (chunks of the longest portion, H * ceil(V / 64), n_seqs), 256 threads
__global__ void __launch_bounds__(256) retention_chunk_out_any_kernel(const RetentionArgs p, const Ragged rg) {
  __shared__ __align__(16) RetTile t;
  __shared__ float P[kRetChunk][kRetChunk + 1];
  const int s = blockIdx.z, c = blockIdx.x, r0 = rg.cu[s] + c * kRetChunk, left = rg.cu[s + 1] - r0;
  if (rg.cu[s + 1] - rg.cu[s] < 2 || left <= 0) return;
  const int n = min(left, kRetChunk), nv = (p.V + 63) / 64, hd = blockIdx.y / nv, v0 = blockIdx.y % nv * 64;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, H = p.H, D = p.D, V = p.V;
  const float* pw = p.pw + (size_t)hd * (kRetChunk + 1);
  const float* q = p.qk + (size_t)r0 * 2 * H * D + (size_t)hd * D;
  const float* k = q + (size_t)H * D;
  const float* v = p.z + (size_t)r0 * p.ldz + 2 * (size_t)H * D + (size_t)hd * V;
  const float* S = p.chunks + ((size_t)(ret_record(rg, s) + c) * H + hd) * D * V;
  float acc[4][4] = {}, st[4][4] = {};
  for (int d0 = 0; d0 < D; d0 += 16) {   // q . k
    for (int e = tid; e < 16 * 64; e += 256) {
      const int r = e >> 4, d = d0 + (e & 15);
      const bool ok = r < n && d < D;
      t.a[e & 15][r] = ok ? q[(size_t)r * 2 * H * D + d] : 0.f;
      t.b[e & 15][r] = ok ? k[(size_t)r * 2 * H * D + d] : 0.f;
    }
    __syncthreads();
    ret_fma(t, tx, ty, acc);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int ri = ty * 4 + i, rj = tx * 4 + j;
      P[ri][rj] = rj <= ri ? acc[i][j] * pw[ri - rj] : 0.f;
      acc[i][j] = 0.f;
    }
  for (int d0 = 0; d0 < D; d0 += 16) {   // q . S
    for (int e = tid; e < 16 * 64; e += 256) {
      const int r = e >> 4, d = d0 + (e & 15), d2 = d0 + (e >> 6), c2 = e & 63;
      t.a[e & 15][r] = (r < n && d < D) ? q[(size_t)r * 2 * H * D + d] : 0.f;
      t.b[e >> 6][c2] = (d2 < D && v0 + c2 < V) ? S[(size_t)d2 * V + v0 + c2] : 0.f;
    }
    __syncthreads();
    ret_fma(t, tx, ty, st);
    __syncthreads();
  }
  for (int j0 = 0; j0 < n; j0 += 16) {   // P . v
    for (int e = tid; e < 16 * 64; e += 256) {
      const int j = j0 + (e >> 6), c2 = e & 63;
      t.a[e >> 6][c2] = P[c2][j];
      t.b[e >> 6][c2] = (j < n && v0 + c2 < V) ? v[(size_t)j * p.ldz + v0 + c2] : 0.f;
    }
    __syncthreads();
    ret_fma(t, tx, ty, acc);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= n) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int vv = v0 + tx * 4 + j;
      if (vv < V) p.o[(size_t)(r0 + r) * H * V + (size_t)hd * V + vv] = fmaf(pw[r + 1], st[i][j], acc[i][j]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ walk over the chunks
constexpr int kRetScanThreads = 128;
// grid (n_seqs, ceil(H D V / (kRetScanThreads VEC))): VEC entries of the state per thread, eight chunks requested at a time
template <int VEC>
__global__ void __launch_bounds__(kRetScanThreads) retention_state_scan_kernel(const RetentionArgs p, const Ragged rg) {
  const int s = blockIdx.x, rows = rg.cu[s + 1] - rg.cu[s];
  const size_t HDV = (size_t)p.H * p.D * p.V, e0 = ((size_t)blockIdx.y * kRetScanThreads + threadIdx.x) * VEC;
  if (rows < 2 || e0 >= HDV) return;
  const float* pw = p.pw + e0 / ((size_t)p.D * p.V) * (kRetChunk + 1);   // (VEC divides V: one head)
  const int nc = (rows + kRetChunk - 1) / kRetChunk;
  const float full = pw[kRetChunk], last = pw[rows - (nc - 1) * kRetChunk];
  float* rec = p.chunks + (size_t)ret_record(rg, s) * HDV + e0;
  float* S_g = p.S + (size_t)rg.slot[s] * p.slot_stride + e0;
  float S[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) S[e] = 0.f;
  if (rg.pos0[s] > 0) ld_vec<VEC>(S_g, S);
  constexpr int kAhead = 8;
  for (int c0 = 0; c0 < nc; c0 += kAhead) {
    float u[kAhead][VEC];
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (c0 + i < nc) ld_vec<VEC>(rec + (size_t)(c0 + i) * HDV, u[i]);
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i >= nc) break;
      st_vec<VEC>(rec + (size_t)(c0 + i) * HDV, S);
      const float a = c0 + i == nc - 1 ? last : full;
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[e] = fmaf(a, S[e], u[i][e]);
    }
  }
  st_vec<VEC>(S_g, S);
}

// ------------------------------------------------------------------------------------------------ tensor-core form
// A ROWS x COLS tile of fp32 rows on its way to two bf16 tiles (x = hi + lo, row stride COLS + 8): `fetch` requests it all (zero beyond
// n rows and `cols` columns), `put` splits it into shared memory, so that a tile's loads run under the products before it
template <int ROWS, int COLS>
struct RetFetch {
  static constexpr int Q = COLS / 4, N = ROWS * Q / 256, LD = COLS + 8;
  static_assert(ROWS * Q % 256 == 0, "whole rounds of 256 threads");
  float f[N][4];
  SSDK_DEVINL void fetch(const float* src, size_t ld, int n, int cols, bool vec) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int e = threadIdx.x + i * 256, r = e / Q, c = e % Q * 4;
      f[i][0] = f[i][1] = f[i][2] = f[i][3] = 0.f;
      if (r < n) {
        if (vec) {
          if (c < cols) ld_vec<4>(src + (size_t)r * ld + c, f[i]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (c + j < cols) f[i][j] = src[(size_t)r * ld + c + j];
        }
      }
    }
  }
  // w (optional): a factor per row, w[r * step]; rows from n on are zero already
  SSDK_DEVINL void put(__nv_bfloat16* hi, __nv_bfloat16* lo, const float* w = nullptr, int step = 0, int n = ROWS) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int e = threadIdx.x + i * 256, r = e / Q, c = e % Q * 4;
      if (w) {
        const float wr = r < n ? w[r * step] : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) f[i][j] *= wr;
      }
      uint32_t h[2], l[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        h[j] = pack_bf16x2(f[i][2 * j], f[i][2 * j + 1]);
        l[j] = pack_bf16x2(f[i][2 * j] - __uint_as_float(h[j] << 16), f[i][2 * j + 1] - __uint_as_float(h[j] & 0xffff0000u));
      }
      *reinterpret_cast<uint2*>(hi + r * LD + c) = make_uint2(h[0], h[1]);
      *reinterpret_cast<uint2*>(lo + r * LD + c) = make_uint2(l[0], l[1]);
    }
  }
};
// c += (ah + al) (bh + bl) without the product of the two low terms
SSDK_DEVINL void ret_mma(float* c, const uint32_t* ah, const uint32_t* al, const uint32_t* bh, const uint32_t* bl) {
  mma_bf16_16816(c, al, bh[0], bh[1]);
  mma_bf16_16816(c, ah, bl[0], bl[1]);
  mma_bf16_16816(c, ah, bh[0], bh[1]);
}

inline size_t ret_state_mma_smem(int KS, int VT) { return (size_t)kRetChunk * 2 * (KS * 16 + 8 + VT * 8 + 8) * 2; }

// grid (chunks of the longest portion, H, n_seqs), 256 threads; D <= 16 KS, V <= 8 VT
template <int KS, int VT>
__global__ void __launch_bounds__(256, 2) retention_chunk_state_mma_kernel(const RetentionArgs p, const Ragged rg) {
  SSDK_DYN_SMEM(uint8_t, rs_sm);
  typedef __nv_bfloat16 T;
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8;
  const int s = blockIdx.z, c = blockIdx.x, hd = blockIdx.y, r0 = rg.cu[s] + c * kRetChunk, left = rg.cu[s + 1] - r0;
  if (rg.cu[s + 1] - rg.cu[s] < 2 || left <= 0) return;
  const int n = min(left, kRetChunk), H = p.H, D = p.D, V = p.V, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  T *kh = (T*)rs_sm, *kl = kh + kRetChunk * LDK, *vh = kl + kRetChunk * LDK, *vl = vh + kRetChunk * LDV;
  {
    RetFetch<kRetChunk, KS * 16> fk;
    RetFetch<kRetChunk, VT * 8> fv;
    fk.fetch(p.qk + (size_t)r0 * 2 * H * D + (size_t)(H + hd) * D, (size_t)2 * H * D, n, D, p.vec);
    fv.fetch(p.z + (size_t)r0 * p.ldz + 2 * (size_t)H * D + (size_t)hd * V, p.ldz, n, V, p.vec);
    fk.put(kh, kl, p.pw + (size_t)hd * (kRetChunk + 1) + n - 1, -1, n);
    fv.put(vh, vl);
  }
  __syncthreads();
  float* out = p.chunks + ((size_t)(ret_record(rg, s) + c) * H + hd) * D * V;
  // operand addresses of this lane: k is read transposed (rows of the result are its columns)
  const int ka = ((lane >> 4) * 8 + (lane & 7)) * LDK + ((lane >> 3) & 1) * 8, va = (((lane >> 3) & 1) * 8 + (lane & 7)) * LDV + (lane >> 4) * 8;
  for (int it = warp; it < KS * (VT / 2); it += 8) {
    const int rt = it % KS, ct = it / KS;
    float acc[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < kRetChunk / 16; ++kk) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      ldmatrix_x4_trans(ah, kh + ka + kk * 16 * LDK + rt * 16);
      ldmatrix_x4_trans(al, kl + ka + kk * 16 * LDK + rt * 16);
      ldmatrix_x4_trans(bh, vh + va + kk * 16 * LDV + ct * 16);
      ldmatrix_x4_trans(bl, vl + va + kk * 16 * LDV + ct * 16);
      ret_mma(acc[0], ah, al, bh, bl);
      ret_mma(acc[1], ah, al, bh + 2, bl + 2);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = rt * 16 + (lane >> 2) + 8 * h, v = ct * 16 + j * 8 + 2 * (lane & 3);
        if (d >= D) continue;
        if (p.vec && v < V) *reinterpret_cast<float2*>(out + (size_t)d * V + v) = make_float2(acc[j][2 * h], acc[j][2 * h + 1]);
        else
          for (int e = 0; e < 2; ++e)
            if (v + e < V) out[(size_t)d * V + v + e] = acc[j][2 * h + e];
      }
  }
}

constexpr int kRetLdP = kRetChunk + 8;
inline size_t ret_out_mma_smem(int KS, int VT) {
  const size_t q = (size_t)kRetChunk * 2 * (KS * 16 + 8) * 2, pk = (size_t)kRetChunk * 2 * kRetLdP * 2;
  return q + (q > pk ? q : pk) + (size_t)kRetChunk * 2 * (VT * 8 + 8) * 2;
}

// grid (chunks of the longest portion, H, n_seqs), 256 threads: warp w has rows 16 (w % 4) .., and of the keys and value columns the half
// w / 4.  Shared memory: q | k, then the decayed scores | a slab of the state, then v (all as two bf16 terms)
template <int KS, int VT>
__global__ void __launch_bounds__(256, 2) retention_chunk_out_mma_kernel(const RetentionArgs p, const Ragged rg) {
  SSDK_DYN_SMEM(uint8_t, ro_sm);
  __shared__ float s_pw[kRetChunk + 1], s_ss[2][kRetChunk];
  typedef __nv_bfloat16 T;
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8, NT = VT / 2, kSlab = KS * 16 < kRetChunk ? KS * 16 : kRetChunk;
  constexpr int kKeep = LDK > kRetLdP ? LDK : kRetLdP;
  const int s = blockIdx.z, c = blockIdx.x, hd = blockIdx.y, r0 = rg.cu[s] + c * kRetChunk, left = rg.cu[s + 1] - r0;
  if (rg.cu[s + 1] - rg.cu[s] < 2 || left <= 0) return;
  const int n = min(left, kRetChunk), H = p.H, D = p.D, V = p.V, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rt = warp & 3, half = warp >> 2;
  T *qh = (T*)ro_sm, *ql = qh + kRetChunk * LDK, *kh = ql + kRetChunk * LDK, *kl = kh + kRetChunk * LDK;
  T *ph = kh, *pl = ph + kRetChunk * kRetLdP;                               // (the scores replace the keys)
  T *vh = kh + 2 * kRetChunk * kKeep, *vl = vh + kRetChunk * LDV;
  const size_t ldq = (size_t)2 * H * D;
  const float* q = p.qk + (size_t)r0 * ldq + (size_t)hd * D;
  if (tid <= kRetChunk) s_pw[tid] = p.pw[(size_t)hd * (kRetChunk + 1) + tid];
  {
    RetFetch<kRetChunk, KS * 16> fq, fk;
    fq.fetch(q, ldq, n, D, p.vec);
    fk.fetch(q + (size_t)H * D, ldq, n, D, p.vec);
    fq.put(qh, ql);
    fk.put(kh, kl);
  }
  // the first slab of the state is on its way under the scores, the next one (at last v) under the products with the one before
  const bool carried = c > 0 || rg.pos0[s] > 0;
  const float* S = p.chunks + ((size_t)(ret_record(rg, s) + c) * H + hd) * D * V;
  const float* v = p.z + (size_t)r0 * p.ldz + 2 * (size_t)H * D + (size_t)hd * V;
  RetFetch<kSlab, VT * 8> fs;
  RetFetch<kRetChunk, VT * 8> fv;
  if (carried) fs.fetch(S, V, D, V, p.vec);
  else fv.fetch(v, p.ldz, n, V, p.vec);
  __syncthreads();
  const int qa = (rt * 16 + (lane & 15)) * LDK + (lane >> 4) * 8;          // this lane's rows of q
  // scores of the warp's 16 rows against its 32 keys
  float sc[4][4] = {};
  if (half * 32 < rt * 16 + 16) {
    const int ka = (half * 32 + (lane >> 4) * 8 + (lane & 7)) * LDK + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      uint32_t ah[4], al[4];
      ldmatrix_x4(ah, qh + qa + k * 16);
      ldmatrix_x4(al, ql + qa + k * 16);
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4(bh, kh + ka + j * 8 * LDK + k * 16);
        ldmatrix_x4(bl, kl + ka + j * 8 * LDK + k * 16);
        ret_mma(sc[j], ah, al, bh, bl);
        ret_mma(sc[j + 1], ah, al, bh + 2, bl + 2);
      }
    }
  }
  __syncthreads();   // every warp has read the keys
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int i = rt * 16 + (lane >> 2) + 8 * h, key = half * 32 + j * 8 + 2 * (lane & 3);
      const float a = key <= i ? sc[j][2 * h] * s_pw[i - key] : 0.f, b = key + 1 <= i ? sc[j][2 * h + 1] * s_pw[i - key - 1] : 0.f;
      const uint32_t hi = pack_bf16x2(a, b);
      *reinterpret_cast<uint32_t*>(ph + i * kRetLdP + key) = hi;
      *reinterpret_cast<uint32_t*>(pl + i * kRetLdP + key) = pack_bf16x2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
    }
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const int va = (((lane >> 3) & 1) * 8 + (lane & 7)) * LDV + (lane >> 4) * 8 + half * NT * 8;   // this lane's rows of a value tile
  if (carried) {   // q . S, a slab of the state's rows at a time
#pragma unroll
    for (int d0 = 0; d0 < KS * 16; d0 += kSlab) {
      if (d0 >= D) break;
      fs.put(vh, vl);
      if (d0 + kSlab < D) fs.fetch(S + (size_t)(d0 + kSlab) * V, V, D - d0 - kSlab, V, p.vec);
      else fv.fetch(v, p.ldz, n, V, p.vec);
      __syncthreads();
#pragma unroll
      for (int k = 0; k < kSlab / 16; ++k) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(ah, qh + qa + d0 + k * 16);
        ldmatrix_x4(al, ql + qa + d0 + k * 16);
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, vh + va + k * 16 * LDV + j * 8);
          ldmatrix_x4_trans(bl, vl + va + k * 16 * LDV + j * 8);
          ret_mma(acc[j], ah, al, bh, bl);
          ret_mma(acc[j + 1], ah, al, bh + 2, bl + 2);
        }
      }
      __syncthreads();
    }
    const float f0 = s_pw[rt * 16 + (lane >> 2) + 1], f1 = s_pw[rt * 16 + (lane >> 2) + 9];
#pragma unroll
    for (int j = 0; j < NT; ++j) { acc[j][0] *= f0; acc[j][1] *= f0; acc[j][2] *= f1; acc[j][3] *= f1; }
  }
  fv.put(vh, vl);
  __syncthreads();
  for (int k = 0; k <= rt; ++k) {   // keys at and before the warp's rows
    uint32_t ah[4], al[4];
    const int pa = (rt * 16 + (lane & 15)) * kRetLdP + (lane >> 4) * 8 + k * 16;
    ldmatrix_x4(ah, ph + pa);
    ldmatrix_x4(al, pl + pa);
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(bh, vh + va + k * 16 * LDV + j * 8);
      ldmatrix_x4_trans(bl, vl + va + k * 16 * LDV + j * 8);
      ret_mma(acc[j], ah, al, bh, bl);
      ret_mma(acc[j + 1], ah, al, bh + 2, bl + 2);
    }
  }
  // unit RMS of every row (its two halves meet in shared memory), gate, rows in the storage type
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NT; ++j) ss = fmaf(acc[j][2 * h], acc[j][2 * h], fmaf(acc[j][2 * h + 1], acc[j][2 * h + 1], ss));   // (columns beyond V are zero)
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if ((lane & 3) == 0) s_ss[half][rt * 16 + (lane >> 2) + 8 * h] = ss;
  }
  __syncthreads();
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int i = rt * 16 + (lane >> 2) + 8 * h;
    if (i >= n) continue;
    const float inv = 1.0f / sqrtf((s_ss[0][i] + s_ss[1][i]) / (float)V + p.eps);
    const float* g = p.z + (size_t)(r0 + i) * p.ldz + 2 * (size_t)H * D + (size_t)H * V + (size_t)hd * V;
    T* y = (T*)p.y + (size_t)(r0 + i) * H * V + (size_t)hd * V;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int v = (half * NT + j) * 8 + 2 * (lane & 3);
      if (p.vec && v < V) {
        const float2 gv = *reinterpret_cast<const float2*>(g + v);
        *reinterpret_cast<uint32_t*>(y + v) = pack_bf16x2(acc[j][2 * h] * inv * gv.x * sigmoid_f(gv.x), acc[j][2 * h + 1] * inv * gv.y * sigmoid_f(gv.y));
      } else {
        for (int e = 0; e < 2; ++e)
          if (v + e < V) y[v + e] = __float2bfloat16_rn(acc[j][2 * h + e] * inv * g[v + e] * sigmoid_f(g[v + e]));
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ single-token rows
constexpr int kRetDecWarps = 8;
inline size_t ret_decode_smem(int D, int V) { return ((size_t)3 * D + V + kRetDecWarps * 128 + 8) * 4; }

// grid (n_seqs, H), kRetDecWarps warps: the warps share the state's rows, a lane has VEC columns of it per step
template <typename T, int VEC>
__global__ void __launch_bounds__(kRetDecWarps * 32) retention_decode_kernel(const RetentionArgs p, const Ragged rg) {
  SSDK_DYN_SMEM(float, rd_sm);
  __shared__ float red[33];
  const int s = blockIdx.x, hd = blockIdx.y, row = rg.cu[s];
  if (rg.cu[s + 1] - row != 1) return;
  const int H = p.H, D = p.D, V = p.V, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, half = (p.inv_freq ? p.rot_dims : 0) >> 1, pos = rg.pos0[s];
  float* part = rd_sm;                          // [warps][128]
  float* q = part + kRetDecWarps * 128;         // [D]
  float* k = q + D;                             // [D]
  float* cs = k + D;                            // [2 half]
  float* o = cs + D;                            // [V]
  const float* z = p.z + (size_t)row * p.ldz;
  const float* v = z + 2 * (size_t)H * D + (size_t)hd * V;
  float* S = p.S + (size_t)rg.slot[s] * p.slot_stride + (size_t)hd * D * V;
  const bool carried = pos > 0;
  // a warp's next kRows rows of the state, columns c .., requested before they are needed: the first under the rotation
  constexpr int kRows = 8;
  float st[kRows][VEC];
  auto fetch = [&](int d0, int c) {
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int d = d0 + i * kRetDecWarps;
#pragma unroll
      for (int e = 0; e < VEC; ++e) st[i][e] = 0.f;
      if (carried && d < D && c < V) ld_vec<VEC>(S + (size_t)d * V + c, st[i]);
    }
  };
  fetch(warp, lane * VEC);
  row_angles(cs, half, pos, p.inv_freq, 1.f);
  __syncthreads();
  if (warp < 2) head_row<float, float, 1>(z + (size_t)(warp * H + hd) * D, warp ? k : q, D, half, cs, (const float*)nullptr, 1.f, warp ? p.k_scale : 1.f, lane);
  __syncthreads();
  const float a = p.pw[(size_t)hd * (kRetChunk + 1) + 1];
  float ss = 0.f;
  for (int v0 = 0; v0 < V; v0 += 32 * VEC) {
    const int c = v0 + lane * VEC;
    float acc[VEC], vv[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) { acc[e] = 0.f; vv[e] = 0.f; }
    if (c < V) {
      ld_vec<VEC>(v + c, vv);
      if (v0 > 0) fetch(warp, c);
      for (int d0 = warp; d0 < D; d0 += kRows * kRetDecWarps) {
#pragma unroll
        for (int i = 0; i < kRows; ++i) {
          const int d = d0 + i * kRetDecWarps;
          if (d >= D) break;
          const float kd = k[d], qd = q[d];
#pragma unroll
          for (int e = 0; e < VEC; ++e) { st[i][e] = fmaf(a, st[i][e], kd * vv[e]); acc[e] = fmaf(qd, st[i][e], acc[e]); }
          st_vec<VEC>(S + (size_t)d * V + c, st[i]);
        }
        if (d0 + kRows * kRetDecWarps < D) fetch(d0 + kRows * kRetDecWarps, c);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) part[warp * 128 + lane * VEC + e] = acc[e];
    __syncthreads();
    for (int j = tid; j < 32 * VEC && v0 + j < V; j += blockDim.x) {
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < kRetDecWarps; ++w) t += part[w * 128 + j];
      o[v0 + j] = t;
      ss = fmaf(t, t, ss);
    }
    __syncthreads();
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)V + p.eps);
  for (int j = tid; j < V; j += blockDim.x) {
    const float g = v[(size_t)H * V + j];
    if (p.o) p.o[(size_t)row * H * V + (size_t)hd * V + j] = o[j];
    st_f<T>((T*)p.y + (size_t)row * H * V + (size_t)hd * V + j, o[j] * inv * g * sigmoid_f(g));
  }
}

}  // namespace ssdk
