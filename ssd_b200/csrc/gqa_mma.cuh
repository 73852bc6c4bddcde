// gqa_mma.cuh — grouped-query attention over the paged cache on the tensor cores (bf16 storage, page rows and heads of whole
// 16-byte pieces, key and value sizes up to 128, up to 16 query heads per key/value head), for the layered (hybrid) models.
// Scores, maxima, sums and the rescaling are fp32; the unnormalised weights are rounded to bf16 for the product with the values.
//
//   gqa_portion_mma_kernel  prompt portions (>= 2 rows), all sequences in one launch: a CTA owns 128 (query, head) rows of one
//                           key/value head and streams the keys its rows see — from the mask's first key of its first query to
//                           its last query — in tiles of 64 (cp.async, two buffers) with an online softmax; no score matrix
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

// 16 query rows (A fragments qf) against NT n-tiles of 8 keys at Ks / Vs (row-major, padded rows); row half h sees the keys
// lo[h] .. hi[h] (positions; key0 is the position of the first key here)
template <int KS, int VT, int NT>
SSDK_DEVINL void gm_keys(const uint32_t (&qf)[KS][4], const __nv_bfloat16* Ks, const __nv_bfloat16* Vs, int key0, const int (&lo)[2], const int (&hi)[2],
                         float scale2, GmRows<VT>& st) {
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
        v = key >= lo[h] && key <= hi[h] ? v * scale2 : -INFINITY;
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

// one tile of keys and values, PER threads per key; keys at and beyond `end` are zero
template <int KS, int VT, int PER>
SSDK_DEVINL void gm_load(const __nv_bfloat16* pool, const Ragged& rg, int s, int g, int G, int D, int V, int key0, int end, __nv_bfloat16* Ks,
                         __nv_bfloat16* Vs) {
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8;
  const int j = threadIdx.x / PER, part = threadIdx.x % PER;
  const bool ok = key0 + j < end;
  const __nv_bfloat16* row = ok ? pool + page_row(rg, s, key0 + j) * (size_t)(G * (D + V)) : pool;
  for (int c = part; c < D / 8; c += PER) cp_async16(Ks + j * LDK + c * 8, row + (ok ? g * D + c * 8 : 0), ok);
  for (int c = part; c < V / 8; c += PER) cp_async16(Vs + j * LDV + c * 8, row + (ok ? G * D + g * V + c * 8 : 0), ok);
  cp_async_commit();
}

inline size_t gm_tile_bytes(int KS, int VT) { return (size_t)kGmKeys * (KS * 16 + 8 + VT * 8 + 8) * 2; }

struct GqaPortionArgs {
  const void* q;      // [G, M, H/G, D] bf16
  const void* cache;  // [rows, G (D + V)] bf16
  void* y;            // [M, H V] bf16
  const float* gate;  // pre-activations of a sigmoid gate, gate[m * ld_gate + h V + v], or nullptr
  int ld_gate;
  int H, G, D, V;
  float scale, sink;
  const void* sinks;  // [H] bf16 learned sink logits (they replace the constant), or nullptr
  KeyMask mask;
};

constexpr int kGpWarps = 8, kGpRows = kGpWarps * 16;

// grid (row tiles of the longest portion, G, n_seqs), 256 threads; the last tiles (most keys) start first
template <int KS, int VT>
__global__ void __launch_bounds__(kGpWarps * 32, 1) gqa_portion_mma_kernel(const GqaPortionArgs p, const Ragged rg) {
  extern __shared__ __align__(16) uint8_t gm_sm[];
  typedef __nv_bfloat16 T;
  constexpr int LDK = KS * 16 + 8, LDV = VT * 8 + 8, kTile = kGmKeys * (LDK + LDV);
  const int g = blockIdx.y, s = blockIdx.z, r0 = rg.cu[s], n = rg.cu[s + 1] - r0, p0 = rg.pos0[s];
  const int hpg = p.H / p.G, rows = n * hpg, row0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kGpRows;
  if (n < 2 || row0 >= rows) return;
  T* sm = (T*)gm_sm;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, D = p.D, V = p.V;
  for (int i = tid; i < 2 * kTile / 2; i += blockDim.x) ((uint32_t*)sm)[i] = 0u;   // columns beyond D and V stay zero
  const int wrow = row0 + warp * 16, wn = min(16, rows - wrow);
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
  const int k_lo = p.mask.first(p0 + row0 / hpg), k_hi = p0 + (min(rows, row0 + kGpRows) - 1) / hpg + 1;
  GmRows<VT> st;
  st.init();
  __syncthreads();
  gm_load<KS, VT, 4>((const T*)p.cache, rg, s, g, p.G, D, V, k_lo, k_hi, sm, sm + kGmKeys * LDK);
  int cur = 0;
  for (int k0 = k_lo; k0 < k_hi; k0 += kGmKeys, cur ^= 1) {
    if (k0 + kGmKeys < k_hi) {
      T* nx = sm + (cur ^ 1) * kTile;
      gm_load<KS, VT, 4>((const T*)p.cache, rg, s, g, p.G, D, V, k0 + kGmKeys, k_hi, nx, nx + kGmKeys * LDK);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (k0 <= w_hi && k0 + kGmKeys > w_lo) {
      const T* Ks = sm + cur * kTile;
      gm_keys<KS, VT, kGmKeys / 8>(qf, Ks, Ks + kGmKeys * LDK, k0, lo, hi, p.scale * kLog2e, st);
    }
    __syncthreads();
  }
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
  const int lo[2] = {k_lo, k_lo}, hi[2] = {k_hi - 1, k_hi - 1};
  __syncthreads();
  if (k_lo < k_hi) gm_load<KS, VT, 2>((const T*)p.cache, rg, s, g, p.G, D, V, k_lo, k_hi, sm, sm + kGmKeys * LDK);
  int cur = 0;
  for (int k0 = k_lo; k0 < k_hi; k0 += kGmKeys, cur ^= 1) {
    if (k0 + kGmKeys < k_hi) {
      T* nx = sm + (cur ^ 1) * kTile;
      gm_load<KS, VT, 2>((const T*)p.cache, rg, s, g, p.G, D, V, k0 + kGmKeys, k_hi, nx, nx + kGmKeys * LDK);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const T* Ks = sm + cur * kTile + warp * 16 * LDK;
    const T* Vs = sm + cur * kTile + kGmKeys * LDK + warp * 16 * LDV;
    gm_keys<KS, VT, 2>(qf, Ks, Vs, k0 + warp * 16, lo, hi, p.scale * kLog2e, st);
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
