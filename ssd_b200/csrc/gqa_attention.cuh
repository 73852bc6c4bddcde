// gqa_attention.cuh — grouped-query causal softmax attention over a paged key/value cache, for the layered (hybrid)
// models.  H query heads share G key/value heads (query head h reads head h / (H / G)); key size D and value size V are
// independent.  A page row holds, for one token, the keys of all G heads (rotated, optionally unit-RMS) and then their
// values: [G D | G V] of storage type T.  The softmax denominator may carry a constant (`sink`: 1 = a sink of score 0
// that has no value) or a learned logit per query head; a key mask limits a query to its last `window` positions (beside the first
// `keep` ones) or to its own chunk of positions.
// Differential attention (maps = 2): every head has two queries and two keys over ONE value head; each map is an attention of its
// own and the head is unit_rms(a1 - lambda a2) (1 - diff).  A page row then holds 2 keys per value head, [head, map] in turn; in the
// kernels G counts keys (2 per value head), H queries, and query (head h, map i) belongs to key 2 (h / (H/G)) + i.
//
//   gqa_prep_kernel      per (token, head): rotation of the first rot_dims dimensions in adjacent or half-apart pairs (angle = position *
//                        frequency in fp32, cos and sin times a constant), optional unit RMS over D; queries go to a
//                        group-major buffer [G, M, H/G, D] (T), keys and raw values into the token's page row
//   gqa_conv_prep_kernel the same behind a short convolution over time of q | k | v (bias, taps, history in the state slot) and an
//                        optional weighted RMS norm over the whole query and key projection, one CTA per row
//   gqa_head_prep_kernel no convolution: weighted RMS norm per head (and map), rotation, cache write, a warp per head of a row
//   kv_gather_kernel     one sequence's pages -> contiguous keys [G, ctx_pad, D] and transposed values [G, V, ctx_pad]
//   portions (>= 2 rows) two batched GEMMs per query block around sink_softmax_kernel (HybRun::gqa_attention)
//   single-token rows    gqa_decode_partial_kernel (all decoding sequences in one launch, context split flash-decoding
//                        style, fp32 weights) + gqa_decode_merge_kernel
//                        (bf16 storage with 16-byte rows: the tensor-core forms of gqa_mma.cuh take both kinds of rows)
//   diff_heads_kernel    group-major fp32 output of the two maps -> [M, H V] (T): the difference, its unit RMS, the constant
//   attn_gate_kernel     group-major fp32 output x sigmoid(gate pre-activation) -> [M, H V] (T) for the output projection
#pragma once
#include "conv_scan.cuh"  // ConvArgs, conv_at
#include "latent_attention.cuh"

namespace ssdk {

struct GqaPrepArgs {
  const float* z; int ldz;     // [M, ldz]: q [H D] | k [G D] | v [G V] (fp32 projections)
  void* q;                     // [G, M, H/G, D] T
  void* cache;                 // [rows, G (D + V)] T (this layer's pool)
  const float* inv_freq;       // [rot_dims / 2] or nullptr
  int H, G, D, V, rot_dims, qk_norm;
  float rot_mult, eps;
  int rot_half;                // 0: entry 2i turns with 2i + 1; 1: entry i turns with i + rot_dims / 2
};

// grid (M, H + G), one warp: units 0 .. H-1 are query heads, H .. H+G-1 key heads (which also copy their value head)
template <typename T>
__global__ void gqa_prep_kernel(const GqaPrepArgs p, const Ragged rg) {
  const int m = blockIdx.x, unit = blockIdx.y, lane = threadIdx.x, s = rg.tok_seq[m];
  const int pos = rg.pos0[s] + (m - rg.cu[s]);
  const int H = p.H, G = p.G, D = p.D, V = p.V;
  const bool is_q = unit < H;
  const int hd = is_q ? unit : unit - H;
  const float* src = p.z + (size_t)m * p.ldz + (is_q ? (size_t)hd * D : (size_t)H * D + (size_t)hd * D);
  T* dst;
  if (is_q) {
    const int hpg = H / G, g = hd / hpg;
    dst = (T*)p.q + (((size_t)g * rg.M + m) * hpg + (hd - g * hpg)) * D;
  } else {
    dst = (T*)p.cache + page_row(rg, s, pos) * (size_t)(G * (D + V)) + (size_t)hd * D;
  }
  // pass 1: rotate pairs, accumulate the square sum; pass 2: scale and store (the pair values are recomputed)
  float ss = 0.f;
  const int rd = p.inv_freq ? p.rot_dims : 0;
  auto value = [&](int d) -> float {
    if (d >= rd) return src[d];
    if (p.rot_half) {
      const int half = rd >> 1, i = d < half ? d : d - half;
      float sn, cs;
      sincosf((float)pos * p.inv_freq[i], &sn, &cs);
      sn *= p.rot_mult; cs *= p.rot_mult;
      return d < half ? src[d] * cs - src[d + half] * sn : src[d] * cs + src[d - half] * sn;
    }
    const int i = d >> 1;
    float sn, cs;
    sincosf((float)pos * p.inv_freq[i], &sn, &cs);
    sn *= p.rot_mult; cs *= p.rot_mult;
    const float a = src[2 * i], b = src[2 * i + 1];
    return (d & 1) ? b * cs + a * sn : a * cs - b * sn;
  };
  float inv = 1.0f;
  if (p.qk_norm) {
    for (int d = lane; d < D; d += 32) { const float v = value(d); ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    inv = 1.0f / sqrtf(ss / (float)D + p.eps);
  }
  for (int d = lane; d < D; d += 32) st_f<T>(dst + d, value(d) * inv);
  if (!is_q) {
    const float* vsrc = p.z + (size_t)m * p.ldz + (size_t)(H + G) * D + (size_t)hd * V;
    T* vdst = (T*)p.cache + page_row(rg, s, pos) * (size_t)(G * (D + V)) + (size_t)G * D + (size_t)hd * V;
    for (int d = lane; d < V; d += 32) st_f<T>(vdst + d, vsrc[d]);
  }
}

struct GqaConvPrepArgs {
  GqaPrepArgs g;               // z / ldz unused: the rows come through the convolution; qk_norm 0 or 2
  ConvArgs conv;               // over the q | k | v columns (C = H D + G D + G V); out / out_t unused, w may be nullptr (one tap of 1)
  const void* norm_w;          // [H D + G D] T weights of the two projection norms (qk_norm == 2)
};

inline size_t gqa_conv_prep_smem(int C, int rot_dims) { return ((size_t)C + rot_dims + 4) * 4; }

// VEC consecutive channels of a row after the convolution.  VEC = 4: channel count, row stride and pointers are whole 16-byte
// pieces and the taps are 2 or 4 (a channel group's taps then are too)
template <typename T, int VEC, int TAPS>
SSDK_DEVINL void conv_group(const ConvArgs& p, const Ragged& rg, int m, int s, int t, int c, float* y) {
  if constexpr (VEC == 1) {
    y[0] = conv_at<T>(p, rg, m, s, t, c);
  } else {
    const bool carried = rg.pos0[s] > 0;
    const float* hist = p.hist + (size_t)rg.slot[s] * p.slot_stride;
    float w[VEC * TAPS], ib[VEC];   // w[e * TAPS + j]: channel c + e, tap j
    ld_contig<T, VEC * TAPS>((const T*)p.w + (size_t)c * TAPS, w);
    if (p.in_bias) ld_contig<T, VEC>((const T*)p.in_bias + c, ib);
#pragma unroll
    for (int e = 0; e < VEC; ++e) y[e] = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int back = TAPS - 1 - j;
      float x[VEC];
      if (back <= t) {
        const float4 f = *reinterpret_cast<const float4*>(p.in + (size_t)(m - back) * p.ld_in + c);
        x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w;
        if (p.in_bias) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) x[e] += ib[e];
        }
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] = carried ? hist[(size_t)(TAPS - 1 - (back - t)) * p.C + c + e] : 0.f;
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = fmaf(w[e * TAPS + j], x[e], y[e]);
    }
  }
}

// grid (M): a CTA convolves the row's q | k | v channels into shared memory, norms the whole query and the whole key
// projection there, turns the first rot_dims entries of every head and stores queries (group-major) and the token's page row.
// VEC = 4: as conv_group, and D, V and the rotated part are multiples of 4 with adjacent pairs.
template <typename T, int VEC, int TAPS>
__global__ void gqa_conv_prep_kernel(const GqaConvPrepArgs p, const Ragged rg) {
  extern __shared__ __align__(16) float gc_sm[];
  __shared__ float red[33];
  const int m = blockIdx.x, s = rg.tok_seq[m], t = m - rg.cu[s], pos = rg.pos0[s] + t;
  const int H = p.g.H, G = p.g.G, D = p.g.D, V = p.g.V, HD = H * D, QK = (H + G) * D, C = QK + G * V;
  const int rd = p.g.inv_freq ? p.g.rot_dims : 0, half = rd >> 1;
  float* y = gc_sm;            // [C]
  float* cs = y + C;           // [half] cos, [half] sin
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, c;
    sincosf((float)pos * p.g.inv_freq[i], &sn, &c);
    cs[i] = c * p.g.rot_mult; cs[half + i] = sn * p.g.rot_mult;
  }
  float sq = 0.f, sk = 0.f;
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    float v[VEC], ss = 0.f;
    conv_group<T, VEC, TAPS>(p.conv, rg, m, s, t, c, v);
    st_vec<VEC>(y + c, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(v[e], v[e], ss);
    if (c < HD) sq += ss;      // (a group of VEC channels never spans q and k: their sizes are multiples of VEC)
    else if (c < QK) sk += ss;
  }
  float iq = 1.f, ik = 1.f;
  const bool norm = p.g.qk_norm == 2;
  if (norm) {
    sq = block_sum(sq, red);
    sk = block_sum(sk, red);
    iq = 1.0f / sqrtf(sq / (float)HD + p.g.eps);
    ik = 1.0f / sqrtf(sk / (float)(G * D) + p.g.eps);
  }
  __syncthreads();
  T* row = (T*)p.g.cache + page_row(rg, s, pos) * (size_t)(G * (D + V));
  const int hpg = H / G;
  const T* nw = (const T*)p.norm_w;
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    float v[VEC];
    ld_vec<VEC>(y + c, v);
    T* dst = row + (c - HD);   // keys of all heads, then values: the page row's own order
    if (c < QK) {
      const int hd = c / D, d = c - hd * D;
      if (norm) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] *= (c < HD ? iq : ik) * ld_f<T>(nw + c + e);
      }
      if (d < rd) {
        if constexpr (VEC == 4) {
#pragma unroll
          for (int e = 0; e < VEC; e += 2) {
            const float co = cs[(d + e) >> 1], sn = cs[half + ((d + e) >> 1)], a = v[e], b = v[e + 1];
            v[e] = a * co - b * sn; v[e + 1] = b * co + a * sn;
          }
        } else {
          const int i = p.g.rot_half ? (d < half ? d : d - half) : d >> 1, step = p.g.rot_half ? half : 1;
          const bool first = p.g.rot_half ? d < half : (d & 1) == 0;
          const int co = first ? c + step : c - step;
          const float o = y[co] * (norm ? (c < HD ? iq : ik) * ld_f<T>(nw + co) : 1.f);   // the other entry of the pair
          v[0] = first ? v[0] * cs[i] - o * cs[half + i] : v[0] * cs[i] + o * cs[half + i];
        }
      }
      if (c < HD) {
        const int g = hd / hpg;
        dst = (T*)p.g.q + (((size_t)g * rg.M + m) * hpg + (hd - g * hpg)) * D + d;
      }
    }
    if constexpr (VEC == 4 && sizeof(T) == 2) {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
      *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) st_f<T>(dst + e, v[e]);
    }
  }
}

// Rows of heads through LANES neighbouring lanes: dst[d] = (rotated) value of src[d] * inv * w[d] * mult, entries d and d + half of the first 2 half
// ones turned by the row's angles (cs: half cosines, then half sines).  VEC = 4: D, half and both pointers are whole groups of four.
template <typename OutT, typename T, int VEC, int LANES = 32>
SSDK_DEVINL void head_row(const float* src, OutT* dst, int D, int half, const float* cs, const T* w, float inv, float mult, int lane) {
  for (int d = lane * VEC; d < D; d += LANES * VEC) {
    float v[VEC];
    ld_vec<VEC>(src + d, v);
    if (w) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] *= inv * ld_f<T>(w + d + e);
    }
    if (d < 2 * half) {
      const bool first = d < half;
      const int od = first ? d + half : d - half, i = first ? d : d - half;
      float o[VEC];
      ld_vec<VEC>(src + od, o);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (w) o[e] *= inv * ld_f<T>(w + od + e);
        v[e] = first ? v[e] * cs[i + e] - o[e] * cs[half + i + e] : v[e] * cs[i + e] + o[e] * cs[half + i + e];
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= mult;
    st_row<OutT, VEC>(dst + d, v);
  }
}

// the row's angles: cs[0 .. half) cosines, cs[half .. 2 half) sines of pos * f_i, times mult
SSDK_DEVINL void row_angles(float* cs, int half, int pos, const float* inv_freq, float mult) {
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, c;
    sincosf((float)pos * inv_freq[i], &sn, &c);
    cs[i] = c * mult; cs[half + i] = sn * mult;
  }
}

struct GqaHeadPrepArgs {
  GqaPrepArgs g;               // H queries and G keys (maps of them per head / value head); qk_norm, rot_half unused
  const void* norm_w;          // [2, D] T: query weight, key weight of the RMS norm over a head's entries, or nullptr
  int maps;
};

// grid (M, y): groups of LANES lanes of a row's CTAs take its H queries, G keys and G / maps values in turn.  dynamic shared memory:
// rot_dims floats
template <typename T, int VEC, int LANES>
__global__ void gqa_head_prep_kernel(const GqaHeadPrepArgs p, const Ragged rg) {
  SSDK_DYN_SMEM(float, hp_cs);
  const int m = blockIdx.x, s = rg.tok_seq[m], pos = rg.pos0[s] + (m - rg.cu[s]), lane = threadIdx.x & (LANES - 1);
  const int H = p.g.H, G = p.g.G, Gv = G / p.maps, D = p.g.D, V = p.g.V, hpg = H / G, half = (p.g.inv_freq ? p.g.rot_dims : 0) >> 1;
  row_angles(hp_cs, half, pos, p.g.inv_freq, p.g.rot_mult);
  __syncthreads();
  const int nw = blockDim.x / LANES;
  const float* z = p.g.z + (size_t)m * p.g.ldz;
  T* row = (T*)p.g.cache + page_row(rg, s, pos) * ((size_t)G * D + (size_t)Gv * V);
  // (every lane of a warp makes the same number of rounds: the sums below are exchanged by all of them)
  for (int u0 = blockIdx.y * nw; u0 < H + G + Gv; u0 += gridDim.y * nw) {
    const int u = u0 + threadIdx.x / LANES;
    float ss = 0.f;
    if (p.norm_w && u < H + G) {
      for (int d = lane * VEC; d < D; d += LANES * VEC) {
        float v[VEC];
        ld_vec<VEC>(z + (size_t)u * D + d, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(v[e], v[e], ss);
      }
    }
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (u >= H + G + Gv) continue;
    if (u >= H + G) {
      const int g = u - H - G;
      head_row<T, T, VEC, LANES>(z + (size_t)(H + G) * D + (size_t)g * V, row + (size_t)G * D + (size_t)g * V, V, 0, hp_cs, (const T*)nullptr, 1.f, 1.f, lane);
      continue;
    }
    const float* src = z + (size_t)u * D;
    const T* w = p.norm_w ? (const T*)p.norm_w + (u < H ? 0 : D) : nullptr;
    const float inv = w ? 1.0f / sqrtf(ss / (float)D + p.g.eps) : 1.f;
    T* dst;
    if (u < H) {
      const int hd = u / p.maps, g = hd / hpg * p.maps + u % p.maps;
      dst = (T*)p.g.q + (((size_t)g * rg.M + m) * hpg + hd % hpg) * D;
    } else {
      dst = row + (size_t)(u - H) * D;
    }
    head_row<T, T, VEC, LANES>(src, dst, D, half, hp_cs, w, inv, 1.f, lane);
  }
}

// grid (ctx_pad): the key of index lo - kept + j of sequence s (KeyMask) -> keys[g][j][:] and vt[g][:][j] (a value head once per map that
// shares it); zero from ctx up to ctx_pad
template <typename T>
__global__ void kv_gather_kernel(const T* __restrict__ cache, T* __restrict__ keys, T* __restrict__ vt, const Ragged rg, int s,
                                 int lo, int kept, int ctx, int ctx_pad, int G, int D, int V, int maps) {
  const int j = blockIdx.x;
  const size_t roww = (size_t)G * D + (size_t)(G / maps) * V;
  const T* row = j < ctx ? cache + page_row(rg, s, key_position(lo - kept + j, lo, kept)) * roww : nullptr;
  for (int i = threadIdx.x; i < G * D; i += blockDim.x) {
    const int g = i / D, d = i - g * D;
    keys[((size_t)g * ctx_pad + j) * D + d] = row ? row[i] : T(0.f);
  }
  for (int i = threadIdx.x; i < G * V; i += blockDim.x) {
    const int g = i / V, v = i - g * V;
    vt[(size_t)i * ctx_pad + j] = row ? row[(size_t)G * D + (size_t)(g / maps) * V + v] : T(0.f);
  }
}

// ---- differential attention: what joins the two maps of a head ----
struct DiffArgs {
  const void* vec;    // [4, D] T: lq1, lk1, lq2, lk2
  int D;
  float diff, eps;
};
// lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, by every warp that needs it
template <typename T>
SSDK_DEVINL float diff_lambda(const DiffArgs& p) {
  const T* v = (const T*)p.vec;
  float a = 0.f, b = 0.f;
  for (int d = threadIdx.x & 31; d < p.D; d += 32) {
    a = fmaf(ld_f<T>(v + d), ld_f<T>(v + p.D + d), a);
    b = fmaf(ld_f<T>(v + 2 * p.D + d), ld_f<T>(v + 3 * p.D + d), b);
  }
  return expf(warp_sum(a)) - expf(warp_sum(b)) + p.diff;
}

// o [G, M, H/G, V] fp32 (G keys = 2 per value head, H queries) -> y [M, (H / 2) V] (T), rows row0 ..; a warp per head.  grid (rows, ceil(H / 2 / warps))
template <typename T>
__global__ void diff_heads_kernel(const float* __restrict__ o, const DiffArgs p, T* __restrict__ y, int M, int H, int G, int V, int row0) {
  const int m = row0 + blockIdx.x, hd = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31, hpg = H / G;
  if (hd >= H / 2) return;
  const float lam = diff_lambda<T>(p);
  const float* a1 = o + (((size_t)(hd / hpg * 2) * M + m) * hpg + hd % hpg) * V;
  const float* a2 = a1 + (size_t)M * hpg * V;
  float ss = 0.f;
  for (int v = lane; v < V; v += 32) { const float x = fmaf(-lam, a2[v], a1[v]); ss = fmaf(x, x, ss); }
  const float f = (1.0f - p.diff) / sqrtf(warp_sum(ss) / (float)V + p.eps);
  for (int v = lane; v < V; v += 32) st_f<T>(y + (size_t)m * (H / 2) * V + (size_t)hd * V + v, fmaf(-lam, a2[v], a1[v]) * f);
}

struct GqaDecodeArgs {
  const void* q;      // [G, M, H/G, D] T
  const void* cache;  // [rows, G D + (G / maps) V] T
  float* part;        // [n_seqs, H, splits, V + 2] fp32: unnormalised P V | running maximum | running sum
  void* y;            // [M, H V] T
  const float* gate;  // pre-activations of a sigmoid gate, gate[m * ld_gate + h V + v], or nullptr
  int ld_gate;
  int H, G, D, V, splits;
  float scale, sink;
  const void* sinks;  // [H] T learned sink logits (they replace the constant), or nullptr
  KeyMask mask;       // keys the token sees
  int maps;           // keys per value head (2: differential attention, joined by gqa_decode_merge_diff_kernel)
  DiffArgs diff;
};

constexpr int kGqaDecWarps = 4;

inline size_t gqa_decode_smem(int D, int V) { return ((size_t)(D + 3) / 4 * 4 + (size_t)kGqaDecWarps * (V + 2)) * 4; }

// grid (n_seqs, H, splits), kGqaDecWarps warps.  A warp takes 32 keys at a time: first every lane scores ONE key (a
// thread-local dot product over D, the key row read in 16-byte pieces where its alignment allows), then every lane owns
// the VPL = ceil(V / 32) value columns lane VPL .. lane VPL + VPL - 1 (one vector load per key) and the 32 weights are
// passed around by shuffle.
template <typename T, int VPL>
__global__ void __launch_bounds__(kGqaDecWarps * 32) gqa_decode_partial_kernel(const GqaDecodeArgs p, const Ragged rg) {
  extern __shared__ __align__(16) float gd_sm[];
  const int s = blockIdx.x, hd = blockIdx.y, sp = blockIdx.z;
  const int row = rg.cu[s];
  if (rg.cu[s + 1] - row != 1) return;
  const int H = p.H, G = p.G, D = p.D, V = p.V, hpg = H / G, g = hd / hpg;
  const int Dp = (D + 3) / 4 * 4;
  float* qs = gd_sm;                      // [Dp] query times scale
  float* wp = gd_sm + Dp;                 // [warps][V + 2]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const T* q = (const T*)p.q + (((size_t)g * rg.M + row) * hpg + (hd - g * hpg)) * D;
  for (int d = tid; d < Dp; d += blockDim.x) qs[d] = d < D ? ld_f<T>(q + d) * p.scale : 0.f;
  __syncthreads();
  int k_lo, k_hi;
  decode_split(rg.pos0[s] + 1, p.mask, sp, p.splits, &k_lo, &k_hi);
  const int first = p.mask.first(rg.pos0[s]), kept = p.mask.kept(first), gv = g / p.maps;
  const size_t roww = (size_t)G * D + (size_t)(G / p.maps) * V;
  constexpr int kPer = 16 / (int)sizeof(T);
  const bool pool16 = ((uintptr_t)p.cache & 15) == 0;
  const bool vec_k = pool16 && D % kPer == 0 && roww % kPer == 0;
  constexpr int kVecBytes = VPL * (int)sizeof(T) >= 16 ? 16 : VPL * (int)sizeof(T);
  constexpr int kVecElems = kVecBytes / (int)sizeof(T);
  const bool vec_v = pool16 && V % VPL == 0 && roww % kVecElems == 0 && ((size_t)G * D) % kVecElems == 0 && V % kVecElems == 0;
  float mx = -INFINITY, sum = 0.f, acc[VPL];
#pragma unroll
  for (int i = 0; i < VPL; ++i) acc[i] = 0.f;
  const int c0 = lane * VPL;  // first value column of this lane
  for (int k0 = k_lo + warp * 32; k0 < k_hi; k0 += kGqaDecWarps * 32) {
    const int key = k0 + lane;
    const bool ok = key < k_hi;
    const size_t prow = ok ? page_row(rg, s, key_position(key, first, kept)) : 0;
    float sc = -INFINITY;
    if (ok) {
      const T* kr = (const T*)p.cache + prow * roww + (size_t)g * D;
      float a0 = 0.f, a1 = 0.f;
      if (vec_k) {
#pragma unroll 4
        for (int d = 0; d < D; d += kPer) {
          float f[kPer];
          ld_contig<T, kPer>(kr + d, f);
#pragma unroll
          for (int e = 0; e < kPer; e += 4) {
            const float4 q4 = *reinterpret_cast<const float4*>(qs + d + e);
            a0 = fmaf(q4.x, f[e], a0); a1 = fmaf(q4.y, f[e + 1], a1); a0 = fmaf(q4.z, f[e + 2], a0); a1 = fmaf(q4.w, f[e + 3], a1);
          }
        }
      } else {
        int d = 0;
        for (; d + 1 < D; d += 2) { a0 = fmaf(qs[d], ld_f<T>(kr + d), a0); a1 = fmaf(qs[d + 1], ld_f<T>(kr + d + 1), a1); }
        if (d < D) a0 = fmaf(qs[d], ld_f<T>(kr + d), a0);
      }
      sc = a0 + a1;
    }
    const float m_new = fmaxf(mx, warp_max(sc));
    const float r = mx == -INFINITY ? 0.f : expf(mx - m_new);
    const float w = ok ? expf(sc - m_new) : 0.f;
    sum = sum * r + warp_sum(w);
#pragma unroll
    for (int i = 0; i < VPL; ++i) acc[i] *= r;
    mx = m_new;
    const int nk = min(32, k_hi - k0);
    // eight keys' value rows are requested before any of them is used
    for (int kk0 = 0; kk0 < nk; kk0 += 8) {
      float f[8][VPL], wk[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int kk = kk0 + u;  // (a lane index below 32 in every case: nk <= 32 and kk0 is a multiple of 8)
        wk[u] = __shfl_sync(0xffffffffu, w, kk);
        const unsigned long long pr = __shfl_sync(0xffffffffu, (unsigned long long)prow, kk);
        const T* vr = (const T*)p.cache + (size_t)pr * roww + (size_t)G * D + (size_t)gv * V + c0;
        const bool live = kk < nk && c0 < V;
        if (live && vec_v) {
          ld_contig<T, VPL>(vr, f[u]);
        } else {
#pragma unroll
          for (int i = 0; i < VPL; ++i) f[u][i] = (live && c0 + i < V) ? ld_f<T>(vr + i) : 0.f;
        }
      }
#pragma unroll
      for (int u = 0; u < 8; ++u)
#pragma unroll
        for (int i = 0; i < VPL; ++i) acc[i] = fmaf(wk[u], f[u][i], acc[i]);
    }
  }
  float* mine = wp + (size_t)warp * (V + 2);
#pragma unroll
  for (int i = 0; i < VPL; ++i)
    if (c0 + i < V) mine[c0 + i] = acc[i];
  if (lane == 0) { mine[V] = mx; mine[V + 1] = sum; }
  __syncthreads();
  // the warps' parts are joined in warp order
  float m = -INFINITY;
  for (int w = 0; w < kGqaDecWarps; ++w) m = fmaxf(m, wp[(size_t)w * (V + 2) + V]);
  float* dst = p.part + (((size_t)s * H + hd) * p.splits + sp) * (V + 2);
  for (int c = tid; c < V + 1; c += blockDim.x) {
    float a = 0.f;
    for (int w = 0; w < kGqaDecWarps; ++w) {
      const float mw = wp[(size_t)w * (V + 2) + V];
      if (mw != -INFINITY) a = fmaf(expf(mw - m), wp[(size_t)w * (V + 2) + (c < V ? c : V + 1)], a);
    }
    dst[c < V ? c : V + 1] = a;
  }
  if (tid == 0) dst[V] = m;
}

constexpr int kGqaMaxSplits = 32;

// grid (n_seqs, H): y = sum_j e^(m_j - m) acc_j / (e^(s - m) + sum_j e^(m_j - m) l_j), s the sink's logit (ln of the constant, or
// the head's learned one), times the sigmoid of the gate's pre-activation if the layer has a gate
template <typename T>
__global__ void gqa_decode_merge_kernel(const GqaDecodeArgs p, const Ragged rg) {
  __shared__ float w[kGqaMaxSplits];
  const int s = blockIdx.x, hd = blockIdx.y;
  const int row = rg.cu[s];
  if (rg.cu[s + 1] - row != 1) return;
  const int V = p.V;
  const float* part = p.part + ((size_t)s * p.H + hd) * p.splits * (V + 2);
  if (threadIdx.x < 32) {   // a lane per split: its weight, normalised
    const int j = threadIdx.x;
    const float sk = p.sinks ? ld_f<T>((const T*)p.sinks + hd) : (p.sink > 0.f ? logf(p.sink) : -INFINITY);
    const float mj = j < p.splits ? part[(size_t)j * (V + 2) + V] : -INFINITY;
    const float m = fmaxf(sk, warp_max(mj));
    const float e = mj == -INFINITY ? 0.f : expf(mj - m);
    const float den = warp_sum(j < p.splits ? e * part[(size_t)j * (V + 2) + V + 1] : 0.f) + (sk == -INFINITY ? 0.f : expf(sk - m));
    w[j] = e / den;
  }
  __syncthreads();
  T* y = (T*)p.y + (size_t)row * p.H * V + (size_t)hd * V;
  for (int c = threadIdx.x; c < V; c += blockDim.x) {
    float a = 0.f;
#pragma unroll 4
    for (int j = 0; j < p.splits; ++j) a = fmaf(w[j], part[(size_t)j * (V + 2) + c], a);
    if (p.gate) a *= sigmoid_f(p.gate[(size_t)row * p.ld_gate + (size_t)hd * V + c]);
    st_f<T>(y + c, a);
  }
}

// grid (n_seqs, H / 2), differential attention: the two maps' splits are joined as above, then with each other.  dynamic shared memory: V floats
template <typename T>
__global__ void gqa_decode_merge_diff_kernel(const GqaDecodeArgs p, const Ragged rg) {
  SSDK_DYN_SMEM(float, md_o);
  __shared__ float w[2][kGqaMaxSplits];
  __shared__ float red[33];
  const int s = blockIdx.x, hd = blockIdx.y, row = rg.cu[s];
  if (rg.cu[s + 1] - row != 1) return;
  const int V = p.V, hpg = p.H / p.G;
  const size_t stride = (size_t)p.splits * (V + 2);
  const float* part = p.part + ((size_t)s * p.H + (size_t)(hd / hpg) * 2 * hpg + hd % hpg) * stride;   // (map 2: hpg heads on)
  if (threadIdx.x < 64) {   // a warp per map, a lane per split: its weight, normalised (the second map's times -lambda)
    const int j = threadIdx.x & 31, map = threadIdx.x >> 5;
    const float* pm = part + map * hpg * stride + (size_t)j * (V + 2) + V;
    const float lam = diff_lambda<T>(p.diff);
    const float mj = j < p.splits ? pm[0] : -INFINITY, m = warp_max(mj);
    const float e = mj == -INFINITY ? 0.f : expf(mj - m);
    const float den = warp_sum(j < p.splits ? e * pm[1] : 0.f);
    w[map][j] = e / den * (map ? -lam : 1.f);
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < V; c += blockDim.x) {
    float a = 0.f, b = 0.f;
#pragma unroll 4
    for (int j = 0; j < p.splits; ++j) {
      a = fmaf(w[0][j], part[(size_t)j * (V + 2) + c], a);
      b = fmaf(w[1][j], part[hpg * stride + (size_t)j * (V + 2) + c], b);
    }
    a += b;
    md_o[c] = a;
    ss = fmaf(a, a, ss);
  }
  ss = block_sum(ss, red);
  const float f = (1.0f - p.diff.diff) / sqrtf(ss / (float)V + p.diff.eps);
  T* y = (T*)p.y + (size_t)row * (p.H / 2) * V + (size_t)hd * V;
  for (int c = threadIdx.x; c < V; c += blockDim.x) st_f<T>(y + c, md_o[c] * f);   // (the thread's own entries)
}

// o [G, M, H/G, V] fp32 (group-major) and gate pre-activations gz[m * ldg + h * V + v] -> y [M, H V] (T) = o * sigmoid(gz), rows row0 ..
template <typename T>
__global__ void attn_gate_kernel(const float* __restrict__ o, const float* __restrict__ gz, int ldg, T* __restrict__ y, int M, int H,
                                 int G, int V, int row0) {
  const int m = row0 + blockIdx.x, hpg = H / G;
  for (int i = threadIdx.x; i < H * V; i += blockDim.x) {
    const int hd = i / V, v = i - hd * V, g = hd / hpg;
    const float ov = o[(((size_t)g * M + m) * hpg + (hd - g * hpg)) * V + v];
    st_f<T>(y + (size_t)m * H * V + i, gz ? ov * sigmoid_f(gz[(size_t)m * ldg + i]) : ov);
  }
}

}  // namespace ssdk
