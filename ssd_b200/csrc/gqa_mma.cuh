// gqa_mma.cuh — grouped-query attention over the paged cache on the tensor cores (bf16 storage, page rows and heads of whole
// 16-byte pieces, key and value sizes up to 128, up to 16 query heads per key/value head), for the layered (hybrid) models.
// Scores, maxima, sums and the rescaling are fp32; the unnormalised weights are rounded to bf16 for the product with the values.
//
//   gqa_portion_mma_kernel  prompt portions (>= 2 rows), all sequences in one launch: a CTA owns 128 (query, head) rows of one
//                           key/value head and streams the keys its rows see — from the mask's first key of its first query to
//                           its last query — in tiles of 64 (cp.async, two buffers) with an online softmax; no score matrix.
//                           Differential attention: the two maps of 64 rows, four warps each, over the same value tile; the maps meet
//                           in shared memory and leave as normed heads
//   gqa_decode_mma_kernel   single-token rows: the heads of a group are the rows of one m16n8k16 tile, the context is split over
//                           CTAs and a tile's 64 keys over the four warps; same partials as gqa_decode_partial_kernel
#pragma once
#include "gqa_attention.cuh"

namespace ssdk {

constexpr int kGmKeys = 64;                       // keys of a tile
constexpr float kLog2e = 1.4426950408889634f, kLn2 = 0.6931471805599453f;

// state of 16 query rows of a warp: a thread holds rows g = lane / 4 and g + 8, and of the value columns 2 (lane % 4), + 1 of
// every n-tile.  Maxima are in units of log2, sums are the thread's own part (joined over the four lanes of a row at the end).
template <int VT>
struct GmRows {
  float m[2], l[2], o[VT][4];
  SSDK_DEVINL void init() {
    m[0] = m[1] = -INFINITY; l[0] = l[1] = 0.f;
#pragma unroll
    for (int v = 0; v < VT; ++v) o[v][0] = o[v][1] = o[v][2] = o[v][3] = 0.f;
  }
};

// 16 query rows (A fragments qf) against NT n-tiles of 8 keys at Ks / Vs (row-major, padded rows); row half h sees the key indices
// lo[h] .. hi[h] and those below kb (KeyMask; key0 is the index of the first key here)
template <int KS, int VT, int NT>
SSDK_DEVINL void gm_keys(const uint32_t (&qf)[KS][4], const __nv_bfloat16* Ks, const __nv_bfloat16* Vs, int key0, const int (&lo)[2], const int (&hi)[2],
                         int kb, float scale2, GmRows<VT>& st) {
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8;
  const int lane = threadIdx.x & 31;
  float s[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
  const __nv_bfloat16* kp = Ks + (size_t)((lane >> 4) * 8 + (lane & 7)) * LDK + ((lane >> 3) & 1) * 8;
#pragma unroll
  for (int k = 0; k < KS; ++k)
#pragma unroll
    for (int n = 0; n < NT; n += 2) {
      uint32_t b[4];
      ldmatrix_x4(b, kp + n * 8 * LDK + k * 16);
      mma_bf16_16816(s[n], qf[k], b[0], b[1]);
      mma_bf16_16816(s[n + 1], qf[k], b[2], b[3]);
    }
  float r[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float mx = st.m[h];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = key0 + n * 8 + 2 * (lane & 3) + e;
        float& v = s[n][2 * h + e];
        v = (key >= lo[h] || key < kb) && key <= hi[h] ? v * scale2 : -INFINITY;
        mx = fmaxf(mx, v);
      }
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    const float ref = mx == -INFINITY ? 0.f : mx;   // (a row that has seen no key yet: everything stays zero)
    r[h] = exp2f(st.m[h] - ref);
    float sum = 0.f;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) { float& v = s[n][2 * h + e]; v = exp2f(v - ref); sum += v; }
    st.l[h] = st.l[h] * r[h] + sum;
    st.m[h] = mx;
  }
#pragma unroll
  for (int v = 0; v < VT; ++v) { st.o[v][0] *= r[0]; st.o[v][1] *= r[0]; st.o[v][2] *= r[1]; st.o[v][3] *= r[1]; }
  const __nv_bfloat16* vp = Vs + (size_t)(((lane >> 3) & 1) * 8 + (lane & 7)) * LDV + (lane >> 4) * 8;
#pragma unroll
  for (int n = 0; n < NT; n += 2) {
    const uint32_t a[4] = {pack_bf16x2(s[n][0], s[n][1]), pack_bf16x2(s[n][2], s[n][3]), pack_bf16x2(s[n + 1][0], s[n + 1][1]),
                           pack_bf16x2(s[n + 1][2], s[n + 1][3])};
#pragma unroll
    for (int v = 0; v < VT; v += 2) {
      uint32_t b[4];
      ldmatrix_x4_trans(b, vp + n * 8 * LDV + v * 8);
      mma_bf16_16816(st.o[v], a, b[0], b[1]);
      mma_bf16_16816(st.o[v + 1], a, b[2], b[3]);
    }
  }
}

// A fragments of 16 query rows of D entries; rows from n on are zero
template <int KS>
SSDK_DEVINL void gm_queries(const __nv_bfloat16* q, int n, int D, uint32_t (&qf)[KS][4]) {
  const int lane = threadIdx.x & 31, g = lane >> 2, t = 2 * (lane & 3);
#pragma unroll
  for (int k = 0; k < KS; ++k)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = g + (i & 1) * 8, d = k * 16 + t + (i >> 1) * 8;
      qf[k][i] = (r < n && d < D) ? *reinterpret_cast<const uint32_t*>(q + (size_t)r * D + d) : 0u;
    }
}

// where a layer's page rows hold key g and its value, and which positions the indices of a query's keys stand for
struct GmPool {
  const __nv_bfloat16* rows;
  int D, V, row_elems, k_off, v_off;   // elements of a page row, offsets of the first key and of the value in it
  int first, kept;                     // KeyMask
};

// one tile of keys (K of them side by side in the page row, each to a tile of its own) and values, PER threads per row; indices at
// and beyond `end` are zero
template <int KS, int VT, int PER, int K = 1>
SSDK_DEVINL void gm_load(const GmPool& p, const Ragged& rg, int s, int key0, int end, __nv_bfloat16* Ks, __nv_bfloat16* Vs) {
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8;
  const int j = threadIdx.x / PER, part = threadIdx.x % PER;
  const bool ok = key0 + j < end;
  const __nv_bfloat16* row = ok ? p.rows + page_row(rg, s, key_position(key0 + j, p.first, p.kept)) * (size_t)p.row_elems : p.rows;
#pragma unroll
  for (int k = 0; k < K; ++k)
    for (int c = part; c < p.D / 8; c += PER) cp_async16(Ks + (k * kGmKeys + j) * LDK + c * 8, row + (ok ? p.k_off + k * p.D + c * 8 : 0), ok);
  for (int c = part; c < p.V / 8; c += PER) cp_async16(Vs + j * LDV + c * 8, row + (ok ? p.v_off + c * 8 : 0), ok);
  cp_async_commit();
}

inline size_t gm_tile_bytes(int KS, int VT, int maps = 1) { return (size_t)kGmKeys * (maps * (KS * 16 + 8) + VT * 8 + 8) * 2; }

struct GqaPortionArgs {
  const void* q;      // [G, M, H/G, D] bf16
  const void* cache;  // [rows, G D + (G / MAPS) V] bf16
  void* y;            // [M, H V] bf16
  const float* gate;  // pre-activations of a sigmoid gate, gate[m * ld_gate + h V + v], or nullptr
  int ld_gate;
  int H, G, D, V;
  float scale, sink;
  const void* sinks;  // [H] bf16 learned sink logits (they replace the constant), or nullptr
  KeyMask mask;
  DiffArgs diff;      // MAPS = 2
};

constexpr int kGpWarps = 8, kGpRows = kGpWarps * 16;

// grid (row tiles of the longest portion, G / MAPS, n_seqs), 256 threads; the last tiles (most keys) start first.  MAPS = 1: 128 rows, 16
// per warp.  MAPS = 2 (differential attention): 64 rows, warps 0 .. 3 take their first map, warps 4 .. 7 the second
template <int KS, int VT, int MAPS>
__global__ void __launch_bounds__(kGpWarps * 32, 1) gqa_portion_mma_kernel(const GqaPortionArgs p, const Ragged rg) {
  extern __shared__ __align__(16) uint8_t gm_sm[];
  typedef __nv_bfloat16 T;
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8, kTile = kGmKeys * (MAPS * LDK + LDV), kRows = kGpRows / MAPS;
  const int gv = blockIdx.y, s = blockIdx.z, r0 = rg.cu[s], n = rg.cu[s + 1] - r0, p0 = rg.pos0[s];
  const int hpg = p.H / p.G, rows = n * hpg, row0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kRows;
  if (n < 2 || row0 >= rows) return;
  T* sm = (T*)gm_sm;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = p.D, V = p.V;
  const int map = MAPS == 1 ? 0 : warp / (kGpWarps / 2), rw = MAPS == 1 ? warp : warp % (kGpWarps / 2), g = gv * MAPS + map;
  for (int i = tid; i < 2 * kTile / 2; i += blockDim.x) ((uint32_t*)sm)[i] = 0u;   // columns beyond D and V stay zero
  const int wrow = row0 + rw * 16, wn = min(16, rows - wrow);
  uint32_t qf[KS][4];
  gm_queries<KS>((const T*)p.q + ((size_t)g * rg.M + r0) * hpg * D + (size_t)(wn > 0 ? wrow : 0) * D, wn, D, qf);
  // positions of this thread's two rows, and what they see; a row outside the portion sees nothing
  int lo[2], hi[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = wrow + (lane >> 2) + 8 * h;
    hi[h] = r < rows ? p0 + r / hpg : -1;
    lo[h] = r < rows ? p.mask.first(hi[h]) : 0;
  }
  const int w_hi = wn > 0 ? p0 + (wrow + wn - 1) / hpg : -1, w_lo = wn > 0 ? p.mask.first(p0 + wrow / hpg) : 0;   // the warp's rows together
  const int first = p.mask.first(p0 + row0 / hpg), kept = p.mask.kept(first), kb = max(p.mask.keep, first);   // every index below kb is a kept key
  const int k_lo = first - kept, k_hi = p0 + (min(rows, row0 + kRows) - 1) / hpg + 1;
  const GmPool pool = {(const T*)p.cache, D, V, p.G * D + p.G / MAPS * V, gv * MAPS * D, p.G * D + gv * V, first, kept};
  GmRows<VT> st;
  st.init();
  __syncthreads();
  gm_load<KS, VT, 4, MAPS>(pool, rg, s, k_lo, k_hi, sm, sm + MAPS * kGmKeys * LDK);
  int cur = 0;
  for (int k0 = k_lo; k0 < k_hi; k0 += kGmKeys, cur ^= 1) {
    if (k0 + kGmKeys < k_hi) {
      T* nx = sm + (cur ^ 1) * kTile;
      gm_load<KS, VT, 4, MAPS>(pool, rg, s, k0 + kGmKeys, k_hi, nx, nx + MAPS * kGmKeys * LDK);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (k0 <= w_hi && (k0 + kGmKeys > w_lo || k0 < kb)) {
      const T* Ks = sm + cur * kTile;
      gm_keys<KS, VT, kGmKeys / 8>(qf, Ks + map * kGmKeys * LDK, Ks + MAPS * kGmKeys * LDK, k0, lo, hi, kb, p.scale * kLog2e, st);
    }
    __syncthreads();
  }
  if constexpr (MAPS == 2) {
    // the second map's rows go through shared memory (fp32, over the tiles), times lambda; the first map's warps finish the heads
    constexpr int LDO = VT * 8 + 4;
    float* o2 = (float*)gm_sm;   // [64][LDO]
    const float lam = diff_lambda<T>(p.diff);
    float inv[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float l = st.l[h];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      inv[h] = 1.0f / l;   // (rows beyond the portion: never used)
      if (map == 1) {
        float* dst = o2 + (size_t)(rw * 16 + (lane >> 2) + 8 * h) * LDO + 2 * (lane & 3);
#pragma unroll
        for (int v = 0; v < VT; ++v) *reinterpret_cast<float2*>(dst + v * 8) = make_float2(st.o[v][2 * h] * inv[h] * lam, st.o[v][2 * h + 1] * inv[h] * lam);
      }
    }
    __syncthreads();
    if (map == 1) return;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = wrow + (lane >> 2) + 8 * h;
      const float* src = o2 + (size_t)(rw * 16 + (lane >> 2) + 8 * h) * LDO + 2 * (lane & 3);
      float ss = 0.f;
#pragma unroll
      for (int v = 0; v < VT; ++v) {
        const float2 b = *reinterpret_cast<const float2*>(src + v * 8);
        float &x = st.o[v][2 * h], &y = st.o[v][2 * h + 1];
        x = fmaf(x, inv[h], -b.x); y = fmaf(y, inv[h], -b.y);
        if (v * 8 + 2 * (lane & 3) < V) ss = fmaf(x, x, fmaf(y, y, ss));
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (r >= rows) continue;
      const float f = (1.0f - p.diff.diff) / sqrtf(ss / (float)V + p.diff.eps);
      T* y = (T*)p.y + (size_t)(r0 + r / hpg) * (p.H / 2) * V + (size_t)(gv * hpg + r % hpg) * V;
#pragma unroll
      for (int v = 0; v < VT; ++v) {
        const int c = v * 8 + 2 * (lane & 3);
        if (c < V) *reinterpret_cast<uint32_t*>(y + c) = pack_bf16x2(st.o[v][2 * h] * f, st.o[v][2 * h + 1] * f);
      }
    }
  } else {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float l = st.l[h];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      const int r = wrow + (lane >> 2) + 8 * h;
      if (r >= rows) continue;
      const int m = r0 + r / hpg, hd = g * hpg + r % hpg;
      if (p.sinks) l += exp2f(ld_f<T>((const T*)p.sinks + hd) * kLog2e - st.m[h]);
      else if (p.sink > 0.f) l += p.sink * exp2f(-st.m[h]);
      const float inv = 1.0f / l;
      T* y = (T*)p.y + (size_t)m * p.H * V + (size_t)hd * V;
      const float* gz = p.gate ? p.gate + (size_t)m * p.ld_gate + (size_t)hd * V : nullptr;
#pragma unroll
      for (int v = 0; v < VT; ++v) {
        const int c = v * 8 + 2 * (lane & 3);
        if (c < V) {
          float a = st.o[v][2 * h] * inv, b = st.o[v][2 * h + 1] * inv;
          if (gz) { a *= sigmoid_f(gz[c]); b *= sigmoid_f(gz[c + 1]); }
          *reinterpret_cast<uint32_t*>(y + c) = pack_bf16x2(a, b);
        }
      }
    }
  }
}

// grid (n_seqs, G, splits), 128 threads: warp w takes keys 16 w .. 16 w + 15 of every tile
template <int KS, int VT>
__global__ void __launch_bounds__(128) gqa_decode_mma_kernel(const GqaDecodeArgs p, const Ragged rg) {
  extern __shared__ __align__(16) uint8_t gm_sm[];
  typedef __nv_bfloat16 T;
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8, kTile = kGmKeys * (LDK + LDV);
  const int s = blockIdx.x, g = blockIdx.y, sp = blockIdx.z, row = rg.cu[s];
  if (rg.cu[s + 1] - row != 1) return;
  T* sm = (T*)gm_sm;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = p.D, V = p.V, hpg = p.H / p.G;
  int k_lo, k_hi;
  decode_split(rg.pos0[s] + 1, p.mask, sp, p.splits, &k_lo, &k_hi);
  for (int i = tid; i < 2 * kTile / 2; i += blockDim.x) ((uint32_t*)sm)[i] = 0u;
  uint32_t qf[KS][4];
  gm_queries<KS>((const T*)p.q + ((size_t)g * rg.M + row) * hpg * D, hpg, D, qf);
  GmRows<VT> st;
  st.init();
  const int lo[2] = {k_lo, k_lo}, hi[2] = {k_hi - 1, k_hi - 1};   // (a split's indices are all seen)
  const int first = p.mask.first(rg.pos0[s]), kept = p.mask.kept(first);
  const GmPool pool = {(const T*)p.cache, D, V, p.G * D + p.G / p.maps * V, g * D, p.G * D + g / p.maps * V, first, kept};
  __syncthreads();
  if (k_lo < k_hi) gm_load<KS, VT, 2>(pool, rg, s, k_lo, k_hi, sm, sm + kGmKeys * LDK);
  int cur = 0;
  for (int k0 = k_lo; k0 < k_hi; k0 += kGmKeys, cur ^= 1) {
    if (k0 + kGmKeys < k_hi) {
      T* nx = sm + (cur ^ 1) * kTile;
      gm_load<KS, VT, 2>(pool, rg, s, k0 + kGmKeys, k_hi, nx, nx + kGmKeys * LDK);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const T* Ks = sm + cur * kTile + warp * 16 * LDK;
    const T* Vs = sm + cur * kTile + kGmKeys * LDK + warp * 16 * LDV;
    gm_keys<KS, VT, 2>(qf, Ks, Vs, k0 + warp * 16, lo, hi, 0, p.scale * kLog2e, st);
    __syncthreads();
  }
  // the warps' parts meet in shared memory and are joined in warp order: [warp][16 rows][V + 2]
  float* wp = (float*)gm_sm;
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float l = st.l[h];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    float* dst = wp + (size_t)(warp * 16 + (lane >> 2) + 8 * h) * (V + 2);
#pragma unroll
    for (int v = 0; v < VT; ++v) {
      const int c = v * 8 + 2 * (lane & 3);
      if (c < V) { dst[c] = st.o[v][2 * h]; dst[c + 1] = st.o[v][2 * h + 1]; }
    }
    if ((lane & 3) == 0) { dst[V] = st.m[h]; dst[V + 1] = l; }
  }
  __syncthreads();
  for (int r = warp; r < hpg; r += 4) {
    float m = -INFINITY, w[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) m = fmaxf(m, wp[(size_t)(x * 16 + r) * (V + 2) + V]);
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const float mx = wp[(size_t)(x * 16 + r) * (V + 2) + V];
      w[x] = mx == -INFINITY ? 0.f : exp2f(mx - m);
    }
    float* dst = p.part + (((size_t)s * p.H + g * hpg + r) * p.splits + sp) * (V + 2);
    for (int c = lane; c < V + 1; c += 32) {
      const int cc = c < V ? c : V + 1;
      float a = 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) a = fmaf(w[x], wp[(size_t)(x * 16 + r) * (V + 2) + cc], a);
      dst[cc] = a;
    }
    if (lane == 0) dst[V] = m == -INFINITY ? m : m * kLn2;
  }
}

inline size_t gqa_decode_mma_smem(int KS, int VT, int V) {
  const size_t tiles = 2 * gm_tile_bytes(KS, VT), join = (size_t)64 * (V + 2) * 4;
  return tiles > join ? tiles : join;
}

}  // namespace ssdk
