// conv_scan.cuh — recurrent mixers that sit behind a short causal convolution, for the layered (hybrid) models.
// Everything here is fp32: the convolution, its activation, gates, decays, step sizes and the carried state; T (bf16 or
// float) is only the storage type of weights and of the rows handed to the next linear layer.
//
//   short_conv_kernel     per-channel causal convolution over time (taps from the checkpoint, last tap = current token),
//                         optional input bias / output bias / SiLU; rows before the portion come from the state slot,
//                         zeros before the sequence
//   conv_state_kernel     saves the last taps - 1 inputs of every sequence's portion into its slot (runs after the readers)
//   input_conv_kernel     a block's input convolutions: y_k = h + conv_k(h) for up to two tap sets over the same rows h (T),
//                         no bias; input_conv_state_kernel saves the last taps - 1 rows of h
//   rglru_scan_kernel     S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,  a_t = exp(-c r_t softplus(lam)),  out = S_t gelu(y_t)
//   selective_scan_kernel S[c,n] = exp(dt_c A[c,n]) S[c,n] + dt_c x_c B_n,  y_c = sum_n S[c,n] C_n + D_c x_c,  out = y silu(z)
//   delta_chunk_prep_kernel  gated delta rule, everything that does not depend on the state: convolution + SiLU of q | k | v,
//                         unit vectors per head, beta, decays per head or per key channel, and per chunk of rows their products
//   delta_chunk_scan_kernel  the walk over the chunks: S = g S; u = beta (v - S^T k); S += k u^T; o = S^T q
//
// A state slot is never cleared: a sequence whose portion starts at position 0 ignores what the slot holds.
#pragma once
#include "layer_ops.cuh"
#include "recurrent.cuh"  // cp_async4

namespace ssdk {

SSDK_DEVINL float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
SSDK_DEVINL float silu_f(float z) { return z * sigmoid_f(z); }
SSDK_DEVINL float gelu_tanh_f(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

struct ConvArgs {
  const float* in;      // [M, ld_in] rows before the convolution; channel c is column c
  int ld_in;
  const void* in_bias;  // [C] T added to every input row (not to the zeros before the sequence), or nullptr
  const void* w;        // [C, taps] T, or nullptr: weight 1 (one tap)
  const void* bias;     // [C] T added to the result, or nullptr
  float* out;           // [M, ld_out] fp32, or nullptr
  int ld_out;
  void* out_t;          // [M, ld_t] T copy for a following linear layer, or nullptr
  int ld_t;
  float* hist;          // state: [taps - 1, C] per slot (with the input bias already added), oldest first
  size_t slot_stride;
  int C, taps;
};

// value of channel c at row m (row t of sequence s) after the convolution, before any activation
template <typename T>
SSDK_DEVINL float conv_at(const ConvArgs& p, const Ragged& rg, int m, int s, int t, int c) {
  float acc = p.bias ? ld_f<T>((const T*)p.bias + c) : 0.f;
  const float ib = p.in_bias ? ld_f<T>((const T*)p.in_bias + c) : 0.f;
  const bool carried = rg.pos0[s] > 0;
  const float* hist = p.hist + (size_t)rg.slot[s] * p.slot_stride;
  for (int j = 0; j < p.taps; ++j) {
    const int back = p.taps - 1 - j;
    float v;
    if (back <= t) v = p.in[(size_t)(m - back) * p.ld_in + c] + ib;
    else v = carried ? hist[(size_t)(p.taps - 1 - (back - t)) * p.C + c] : 0.f;
    acc = fmaf(p.w ? ld_f<T>((const T*)p.w + (size_t)c * p.taps + j) : 1.f, v, acc);
  }
  return acc;
}

// ACT: 0 none, 1 SiLU.  grid (M, ceil(C / blockDim))
template <typename T, int ACT>
__global__ void short_conv_kernel(const ConvArgs p, const Ragged rg) {
  const int m = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.C) return;
  const int s = rg.tok_seq[m];
  float v = conv_at<T>(p, rg, m, s, m - rg.cu[s], c);
  if (ACT == 1) v = silu_f(v);
  if (p.out) p.out[(size_t)m * p.ld_out + c] = v;
  if (p.out_t) st_f<T>((T*)p.out_t + (size_t)m * p.ld_t + c, v);
}

// grid (n_seqs, ceil(C / blockDim)).  New history = the last taps - 1 entries of (old history ++ this portion's inputs);
// entry j is read from an index above j, so one thread per channel may work in place in ascending order.
template <typename T>
__global__ void conv_state_kernel(const ConvArgs p, const Ragged rg) {
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.C) return;
  const int r0 = rg.cu[s], n = rg.cu[s + 1] - r0, keep = p.taps - 1;
  const bool carried = rg.pos0[s] > 0;
  const float ib = p.in_bias ? ld_f<T>((const T*)p.in_bias + c) : 0.f;
  float* hist = p.hist + (size_t)rg.slot[s] * p.slot_stride;
  for (int j = 0; j < keep; ++j) {
    const int idx = n + j;
    float v;
    if (idx < keep) v = carried ? hist[(size_t)idx * p.C + c] : 0.f;
    else v = p.in[(size_t)(r0 + idx - keep) * p.ld_in + c] + ib;
    hist[(size_t)j * p.C + c] = v;
  }
}

// Residual input convolution of a block's sublayers.  h [M, C] (T) are the rows both sublayers read; sublayer k gets
// y_k[m, c] = h[m, c] + sum_j w_k[c, j] h[row of position t - taps + 1 + j, c] with zeros before the sequence's start and the
// rows before the portion taken from the state slot (hist [taps - 1, C] fp32 per slot, oldest first).  Sums in fp32.
struct InputConvArgs {
  const void* h;        // [M, C] T
  const void* w;        // [2, C, taps] T: taps of y1, then of y2
  void* y1;             // [M, C] T
  void* y2;             // [M, C] T or nullptr
  float* hist; size_t slot_stride;
  int C, taps;
};

// grid (M, ceil(C / blockDim)): one channel per thread, any number of taps
template <typename T>
__global__ void input_conv_kernel(const InputConvArgs p, const Ragged rg) {
  const int m = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.C) return;
  const int s = rg.tok_seq[m], t = m - rg.cu[s];
  const bool carried = rg.pos0[s] > 0;
  const float* hist = p.hist + (size_t)rg.slot[s] * p.slot_stride;
  const T* h = (const T*)p.h;
  const T* w1 = (const T*)p.w + (size_t)c * p.taps;
  const T* w2 = w1 + (size_t)p.C * p.taps;
  const float cur = ld_f<T>(h + (size_t)m * p.C + c);
  float a1 = 0.f, a2 = 0.f;
  for (int j = 0; j < p.taps; ++j) {
    const int back = p.taps - 1 - j;
    float v;
    if (back == 0) v = cur;
    else if (back <= t) v = ld_f<T>(h + (size_t)(m - back) * p.C + c);
    else v = carried ? hist[(size_t)(p.taps - 1 - (back - t)) * p.C + c] : 0.f;
    a1 = fmaf(ld_f<T>(w1 + j), v, a1);
    if (p.y2) a2 = fmaf(ld_f<T>(w2 + j), v, a2);
  }
  st_f<T>((T*)p.y1 + (size_t)m * p.C + c, cur + a1);
  if (p.y2) st_f<T>((T*)p.y2 + (size_t)m * p.C + c, cur + a2);
}

// The same with 16 bytes of channels per thread (8 bf16 or 4 floats) and the taps in registers: C a multiple of that,
// rows and taps 16-byte aligned.  grid (M, ceil(C / VEC / blockDim)).  Same sums in the same order as the scalar form.
template <typename T, int TAPS>
__global__ void input_conv_vec_kernel(const InputConvArgs p, const Ragged rg) {
  constexpr int VEC = 16 / (int)sizeof(T);
  const int m = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= p.C) return;
  const int s = rg.tok_seq[m], t = m - rg.cu[s];
  const bool carried = rg.pos0[s] > 0;
  const float* hist = p.hist + (size_t)rg.slot[s] * p.slot_stride;
  const T* h = (const T*)p.h;
  float w1[VEC * TAPS], w2[VEC * TAPS];   // entry e * TAPS + j: channel c + e, tap j
  ld_contig<T, VEC * TAPS>((const T*)p.w + (size_t)c * TAPS, w1);
  if (p.y2) ld_contig<T, VEC * TAPS>((const T*)p.w + ((size_t)p.C + c) * TAPS, w2);
  float cur[VEC], a1[VEC], a2[VEC];
  ld_contig<T, VEC>(h + (size_t)m * p.C + c, cur);
#pragma unroll
  for (int e = 0; e < VEC; ++e) a1[e] = a2[e] = 0.f;
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    const int back = TAPS - 1 - j;
    float v[VEC];
    if (back == 0) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = cur[e];
    } else if (back <= t) {
      ld_contig<T, VEC>(h + (size_t)(m - back) * p.C + c, v);
    } else if (carried) {
      ld_contig<float, VEC>(hist + (size_t)(TAPS - 1 - (back - t)) * p.C + c, v);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = 0.f;
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      a1[e] = fmaf(w1[e * TAPS + j], v[e], a1[e]);
      if (p.y2) a2[e] = fmaf(w2[e * TAPS + j], v[e], a2[e]);
    }
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) { a1[e] += cur[e]; a2[e] += cur[e]; }
  st_contig<T, VEC>((T*)p.y1 + (size_t)m * p.C + c, a1);
  if (p.y2) st_contig<T, VEC>((T*)p.y2 + (size_t)m * p.C + c, a2);
}

// grid (n_seqs, ceil(C / blockDim)); runs after input_conv_kernel.  As conv_state_kernel: entry j is read from an index
// above j, so one thread per channel works in place in ascending order.
template <typename T>
__global__ void input_conv_state_kernel(const InputConvArgs p, const Ragged rg) {
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.C) return;
  const int r0 = rg.cu[s], n = rg.cu[s + 1] - r0, keep = p.taps - 1;
  const bool carried = rg.pos0[s] > 0;
  float* hist = p.hist + (size_t)rg.slot[s] * p.slot_stride;
  for (int j = 0; j < keep; ++j) {
    const int idx = n + j;
    float v;
    if (idx < keep) v = carried ? hist[(size_t)idx * p.C + c] : 0.f;
    else v = ld_f<T>((const T*)p.h + (size_t)(r0 + idx - keep) * p.C + c);
    hist[(size_t)j * p.C + c] = v;
  }
}

// fp32 columns -> T columns (operand of a following linear layer)
template <typename T>
__global__ void cast_cols_kernel(const float* __restrict__ src, int ld_src, T* __restrict__ dst, int ld_dst, int cols) {
  const int m = blockIdx.x;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) st_f<T>(dst + (size_t)m * ld_dst + c, src[(size_t)m * ld_src + c]);
}

// ---------------------------------------------------------------------------------------------- rglru
struct RglruArgs {
  const float* u; int ld_u;          // [M, R] convolved x branch
  const float* gates; int ld_g;      // [M, blocks * 2 bs]: per block recurrence-gate slots, then input-gate slots
                                     // (pre-activations before rglru_gate_kernel, decay a and input term b after it)
  const void* gate_bias;             // [blocks, 2 bs] T
  const void* lam;                   // [R] T
  const float* y; int ld_y;          // [M, ...] y branch (pre-activation before rglru_gate_kernel, gelu after)
  const void* y_bias;                // [R] T
  void* out;                         // [M, R] T: S * gelu_tanh(y)
  float* S; size_t slot_stride;      // [R] per slot
  int R, bs;
  float decay_mult;
};

// grid (M, ceil(R / blockDim)): everything of a row that does not depend on the state, for all rows at once and in place:
// gates[m][recurrence slot] <- a = exp(-c r softplus(lam)), gates[m][input slot] <- sqrt(1 - a^2) i u,
// y[m] <- gelu_tanh(y[m] + bias)
template <typename T>
__global__ void rglru_gate_kernel(const RglruArgs p, float* __restrict__ gates, float* __restrict__ y) {
  const int m = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.R) return;
  const int b = c / p.bs, cb = c - b * p.bs;
  const int gr = b * 2 * p.bs + cb, gi = gr + p.bs;
  const float sp = softplus_f(ld_f<T>((const T*)p.lam + c)) * p.decay_mult;
  float* grow = gates + (size_t)m * p.ld_g;
  const float log_a = -sigmoid_f(grow[gr] + ld_f<T>((const T*)p.gate_bias + gr)) * sp;
  const float i = sigmoid_f(grow[gi] + ld_f<T>((const T*)p.gate_bias + gi));
  grow[gr] = expf(log_a);
  // 1 - a^2 through expm1: exact also where a is within an ulp of 1
  grow[gi] = sqrtf(-expm1f(2.0f * log_a)) * i * p.u[(size_t)m * p.ld_u + c];
  float* yp = y + (size_t)m * p.ld_y + c;
  *yp = gelu_tanh_f(*yp + ld_f<T>((const T*)p.y_bias + c));
}

constexpr int kRglruRows = 16;  // rows whose operands are requested together

// grid (n_seqs, ceil(R / blockDim)): one thread per channel walks its sequence's rows, S = a S + b, out = S y, with the
// operands rglru_gate_kernel left (sixteen rows' loads in flight at a time).
template <typename T>
__global__ void rglru_scan_kernel(const RglruArgs p, const Ragged rg) {
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= p.R) return;
  const int b = c / p.bs, cb = c - b * p.bs;
  const int gr = b * 2 * p.bs + cb, gi = gr + p.bs;
  float* Sp = p.S + (size_t)rg.slot[s] * p.slot_stride + c;
  float S = rg.pos0[s] > 0 ? *Sp : 0.f;
  const int r0 = rg.cu[s], r1 = rg.cu[s + 1];
  for (int m0 = r0; m0 < r1; m0 += kRglruRows) {
    float a[kRglruRows], bb[kRglruRows], y[kRglruRows];
#pragma unroll
    for (int k = 0; k < kRglruRows; ++k) {
      const int m = min(m0 + k, r1 - 1);
      a[k] = p.gates[(size_t)m * p.ld_g + gr]; bb[k] = p.gates[(size_t)m * p.ld_g + gi]; y[k] = p.y[(size_t)m * p.ld_y + c];
    }
#pragma unroll
    for (int k = 0; k < kRglruRows; ++k) {
      if (m0 + k < r1) {
        S = fmaf(a[k], S, bb[k]);
        st_f<T>((T*)p.out + (size_t)(m0 + k) * p.R + c, S * y[k]);
      }
    }
  }
  *Sp = S;
}

// ---------------------------------------------------------------------------------------------- selective scan
struct SelScanArgs {
  const float* x; int ld_x;          // [M, inner] convolved, SiLU'd input
  const float* dtz; int ld_dt;       // [M, inner] step sizes (after softplus)
  const float* bc; int ld_bc;        // [M, ...]: B in columns [0, N), C in [N, 2N)
  const void* A_log;                 // [inner, N] T
  const void* Dw;                    // [inner] T
  const float* z; int ld_z;          // [M, inner] gate values silu(z)
  void* out;                         // [M, inner] T: y * silu(z)
  float* S; size_t slot_stride;      // [inner, N] per slot
  int inner, N;
};

// grid (M, ceil(inner / blockDim)): the state-independent part of a row, in place: dtz <- softplus(dtz + bias), z <- silu(z)
template <typename T>
__global__ void selective_gate_kernel(float* __restrict__ dtz, int ld_dt, const T* __restrict__ dt_bias, float* __restrict__ z, int ld_z,
                                      int inner) {
  const int m = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= inner) return;
  float* d = dtz + (size_t)m * ld_dt + c;
  *d = softplus_f(*d + ld_f<T>(dt_bias + c));
  float* zp = z + (size_t)m * ld_z + c;
  *zp = silu_f(*zp);
}

constexpr int kSelRows = 8;  // rows whose inputs are requested (and whose B | C are staged) together

// A channel's N states are spread over LPC = blockDim.x lanes of a warp (a power of two), NT states per lane in
// registers (N <= NT * LPC); blockDim.y channels per CTA, grid (n_seqs, ceil(inner / blockDim.y)).  Per row a lane
// advances its states and the lanes' parts of y = sum_n S[n] C[n] meet by shuffle (a fixed tree).  exp(dt A) is taken as
// exp2(dt (A log2 e)).  dtz holds the step sizes and z the gate values selective_gate_kernel left.  NT == 0: any N, one
// lane per channel, the state stays in its slot (global memory).  dynamic shared memory: kSelRows * 2 N floats.
template <typename T, int NT>
__global__ void selective_scan_kernel(const SelScanArgs p, const Ragged rg) {
  extern __shared__ float sel_sm[];
  const int s = blockIdx.x, lpc = blockDim.x, ln = threadIdx.x, N = p.N;
  const int c = blockIdx.y * blockDim.y + threadIdx.y, tid = threadIdx.y * lpc + ln, nthr = lpc * blockDim.y;
  const bool live = c < p.inner;
  const bool carried = rg.pos0[s] > 0;
  const int n0 = ln * NT;  // first state of this lane
  float A2[NT > 0 ? NT : 1], S[NT > 0 ? NT : 1];
  float* Sg = p.S + (size_t)rg.slot[s] * p.slot_stride + (size_t)(live ? c : 0) * N;
  if (NT > 0) {
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const bool ok = live && n0 + n < N;
      A2[n] = ok ? -expf(ld_f<T>((const T*)p.A_log + (size_t)c * N + n0 + n)) * 1.4426950408889634f : 0.f;
      S[n] = (ok && carried) ? Sg[n0 + n] : 0.f;
    }
  } else if (live && !carried) {
    for (int n = 0; n < N; ++n) Sg[n] = 0.f;
  }
  const float Dc = live ? ld_f<T>((const T*)p.Dw + c) : 0.f;
  const int r0 = rg.cu[s], r1 = rg.cu[s + 1], cc = live ? c : 0;
  for (int m0 = r0; m0 < r1; m0 += kSelRows) {
    const int nr = min(kSelRows, r1 - m0);
    float dt[kSelRows], xv[kSelRows], zv[kSelRows];
#pragma unroll
    for (int r = 0; r < kSelRows; ++r) {
      const int m = min(m0 + r, r1 - 1);
      dt[r] = p.dtz[(size_t)m * p.ld_dt + cc]; xv[r] = p.x[(size_t)m * p.ld_x + cc]; zv[r] = p.z[(size_t)m * p.ld_z + cc];
    }
    __syncthreads();
    for (int i = tid; i < nr * 2 * N; i += nthr) {
      const int r = i / (2 * N), k = i - r * 2 * N;
      sel_sm[i] = p.bc[(size_t)(m0 + r) * p.ld_bc + k];
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < kSelRows; ++r) {
      if (r < nr) {
        const int m = m0 + r;
        const float dx = dt[r] * xv[r];
        const float* B = sel_sm + r * 2 * N;
        const float* Cm = B + N;
        float y = 0.f;
        if (NT > 0) {
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            if (n0 + n < N) {
              S[n] = fmaf(exp2f(dt[r] * A2[n]), S[n], dx * B[n0 + n]);
              y = fmaf(S[n], Cm[n0 + n], y);
            }
          }
          for (int o = lpc >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        } else if (live) {
          for (int n = 0; n < N; ++n) {
            const float a = -expf(ld_f<T>((const T*)p.A_log + (size_t)c * N + n));
            const float sn = fmaf(expf(dt[r] * a), Sg[n], dx * B[n]);
            Sg[n] = sn;
            y = fmaf(sn, Cm[n], y);
          }
        }
        if (live && ln == 0) st_f<T>((T*)p.out + (size_t)m * p.inner + c, fmaf(Dc, xv[r], y) * zv[r]);
      }
    }
  }
  if (NT > 0 && live) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
      if (n0 + n < N) Sg[n0 + n] = S[n];
  }
}

// ---------------------------------------------------------------------------------------------- gated delta rule
// Per head, S [D, V]:  S = diag(g_t) S;  u_t = beta_t (v_t - S^T k_t);  S += k_t u_t^T;  o_t = S^T q_t.
// C consecutive rows (a chunk) are taken together.  With S the state before the chunk, G_i = g_1 .. g_i (per key channel) and
// G_(j,i] = g_(j+1) .. g_i, unrolling the recurrence gives
//     u_i = beta_i (v_i - (G_i k_i)^T S - sum_{j<i} A_ij u_j),         A_ij = sum_d k_i G_(j,i] k_j
//     o_i = (G_i q_i)^T S + sum_{j<=i} B_ij u_j,                       B_ij = sum_d q_i G_(j,i] k_j
//     S  <- S + (G_C - 1) S + sum_i (G_(i,C] k_i) u_i^T
// A, B and every scaled k and q are independent of the state, and so is X = (I + diag(beta) A)^-1 diag(beta) (unit triangular
// inverse): u = X r and o = (G q)^T S + (B X) r with r_i = v_i - (G_i k_i)^T S.  delta_chunk_prep_kernel makes them for all
// chunks at once, delta_chunk_scan_kernel walks the chunks.  No quotient of decays is formed, so any decay in (0, 1] is safe;
// the factor that survives from chunk to chunk, G_C - 1, comes from expm1 of the summed log decays.  All fp32.
//
// Record of one (chunk, head), DP >= D padded with zeros:  G k [C][DP] | G_(.,C] k [C][DP] | G q [C][DP] | G_C - 1 [DP] |
// X [C][C] | B X [C][C] (C = 1: padded to 4 floats).  Rows behind the portion's end are zero.
inline __host__ __device__ int delta_record(int DP, int C) { return (3 * C + 1) * DP + (C > 1 ? 2 * C * C : 4); }

constexpr int kDeltaChunk = 8;   // rows of a chunk (1 in calls that bring one row per sequence)
constexpr int kDeltaTaps = 4;    // convolutions up to this length keep their rows in registers

struct DeltaPrepArgs {
  ConvArgs conv;          // over the q | k | v columns (C = 2 G D + H V); out / out_t unused
  const float* b; int ld_b;    // [M, ...]: beta pre-activations in columns [0, H)
  const float* a; int ld_a;    // decay pre-activations: [M, ...] columns [0, H), or (per_channel) [M, H D]
  const void* A_log;      // [H] T
  const void* dt_bias;    // [H] T, or (per_channel) [H D]
  float* v;               // [M, H V]
  float* rec;             // records, (chunk index, head)
  int H, G, D, V, DP, per_channel;
  float q_scale, unit_eps;
};

// chunk ci of sequence s: records of different sequences never overlap (a portion of n rows has at most n / C + 1 chunks)
SSDK_DEVINL size_t delta_chunk_index(const Ragged& rg, int s, int ci, int C) { return (size_t)(rg.cu[s] / C + s + ci); }

// channel c of the convolution at C consecutive rows t0 .. of sequence s (rows from nr on: zero), then SiLU
template <typename T, int C>
SSDK_DEVINL void conv_silu_rows(const ConvArgs& p, const Ragged& rg, int s, int t0, int nr, int c, float* y) {
  const int r0 = rg.cu[s];
  if (p.taps > kDeltaTaps) {
#pragma unroll
    for (int i = 0; i < C; ++i) y[i] = i < nr ? silu_f(conv_at<T>(p, rg, r0 + t0 + i, s, t0 + i, c)) : 0.f;
    return;
  }
  const bool carried = rg.pos0[s] > 0;
  const float* hist = p.hist + (size_t)rg.slot[s] * p.slot_stride;
  float w[kDeltaTaps], x[C + kDeltaTaps - 1];   // w[b]: weight of the row b steps back; x[i + kDeltaTaps - 1]: row t0 + i
#pragma unroll
  for (int b = 0; b < kDeltaTaps; ++b) w[b] = b < p.taps ? ld_f<T>((const T*)p.w + (size_t)c * p.taps + (p.taps - 1 - b)) : 0.f;
#pragma unroll
  for (int i = 1 - kDeltaTaps; i < C; ++i) {
    const int t = t0 + i;
    float v = 0.f;
    if (i > -p.taps && i < nr) {
      if (t >= 0) v = p.in[(size_t)(r0 + t) * p.ld_in + c];
      else if (carried) v = hist[(size_t)(p.taps - 1 + t) * p.C + c];
    }
    x[i + kDeltaTaps - 1] = v;
  }
#pragma unroll
  for (int i = 0; i < C; ++i) {
    float acc = 0.f;
#pragma unroll
    for (int b = kDeltaTaps - 1; b >= 0; --b) acc = fmaf(w[b], x[i - b + kDeltaTaps - 1], acc);
    y[i] = i < nr ? silu_f(acc) : 0.f;
  }
}

inline size_t delta_prep_smem(int D, int C) { return ((size_t)3 * C * D + 3 * C * C + 3 * C + 4) * 4; }

// grid (chunks of the longest portion, n_seqs, H), 128 threads
template <typename T, int C>
__global__ void __launch_bounds__(128) delta_chunk_prep_kernel(const DeltaPrepArgs p, const Ragged rg) {
  extern __shared__ float dp_sm[];
  constexpr int kThreads = 128, kSlices = kThreads / C;
  const int ci = blockIdx.x, s = blockIdx.y, h = blockIdx.z, t0 = ci * C, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int m0 = rg.cu[s] + t0, nr = min(C, rg.cu[s + 1] - m0);
  if (nr <= 0) return;
  const int D = p.D, V = p.V, DP = p.DP, GD = p.G * D, g = h / (p.H / p.G);
  float* kk = dp_sm;                // [C][D] keys, then unit keys
  float* qq = kk + C * D;           // [C][D]
  float* ll = qq + C * D;           // [C][D] log decays, then decays
  float* A = ll + C * D;            // [C][C]
  float* B = A + C * C;             // [C][C]
  float* X = B + C * C;             // [C][C]
  float* sc = X + C * C;            // [2 C] 1 / length of the keys, then of the queries
  float* beta = sc + 2 * C;         // [C]
  float* rec = p.rec + (delta_chunk_index(rg, s, ci, C) * p.H + h) * delta_record(DP, C);
  const float rate = -expf(ld_f<T>((const T*)p.A_log + h));
  for (int d = tid; d < D; d += kThreads) {
    float y[C];
    conv_silu_rows<T, C>(p.conv, rg, s, t0, nr, g * D + d, y);
#pragma unroll
    for (int i = 0; i < C; ++i) qq[i * D + d] = y[i];
    conv_silu_rows<T, C>(p.conv, rg, s, t0, nr, GD + g * D + d, y);
    const int c = p.per_channel ? h * D + d : h;
    const float bias = ld_f<T>((const T*)p.dt_bias + c);
#pragma unroll
    for (int i = 0; i < C; ++i) {
      kk[i * D + d] = y[i];
      ll[i * D + d] = i < nr ? rate * softplus_f(p.a[(size_t)(m0 + i) * p.ld_a + c] + bias) : 0.f;
    }
  }
  for (int d = tid; d < V; d += kThreads) {
    float y[C];
    conv_silu_rows<T, C>(p.conv, rg, s, t0, nr, 2 * GD + h * V + d, y);
#pragma unroll
    for (int i = 0; i < C; ++i)
      if (i < nr) p.v[((size_t)(m0 + i) * p.H + h) * V + d] = y[i];
  }
  if (tid < C) beta[tid] = tid < nr ? sigmoid_f(p.b[(size_t)(m0 + tid) * p.ld_b + h]) : 0.f;
  __syncthreads();
  for (int x = warp; x < 2 * C; x += kThreads / 32) {   // (kk and qq are adjacent: row x of the two)
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) { const float v = kk[x * D + d]; ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    if (lane == 0) sc[x] = (x < C ? 1.0f : p.q_scale) / sqrtf(ss + p.unit_eps);
  }
  __syncthreads();
  for (int d = tid; d < DP; d += kThreads) {
    float k[C], e[C], L = 0.f, G = 1.f;
#pragma unroll
    for (int i = 0; i < C; ++i) {
      float q = 0.f;
      k[i] = 0.f; e[i] = 1.f;
      if (d < D) {
        const float l = ll[i * D + d];
        k[i] = kk[i * D + d] * sc[i]; q = qq[i * D + d] * sc[C + i]; e[i] = expf(l);
        kk[i * D + d] = k[i]; qq[i * D + d] = q; ll[i * D + d] = e[i];
        L += l;
      }
      G *= e[i];
      rec[i * DP + d] = k[i] * G;
      rec[(2 * C + i) * DP + d] = q * G;
    }
    G = 1.f;
#pragma unroll
    for (int i = C - 1; i >= 0; --i) { rec[(C + i) * DP + d] = k[i] * G; G *= e[i]; }
    rec[3 * C * DP + d] = expm1f(L);
  }
  __syncthreads();
  {
    const int jj = tid / kSlices, sl = tid % kSlices;   // key row jj, channels sl, sl + kSlices, ..
    float a[C], b[C];
#pragma unroll
    for (int i = 0; i < C; ++i) a[i] = b[i] = 0.f;
    for (int d = sl; d < D; d += kSlices) {
      float run = kk[jj * D + d];
#pragma unroll
      for (int i = 0; i < C; ++i) {
        if (i > jj) { run *= ll[i * D + d]; a[i] = fmaf(kk[i * D + d], run, a[i]); }
        if (i >= jj) b[i] = fmaf(qq[i * D + d], run, b[i]);
      }
    }
    if constexpr (C == 1) {
      b[0] = warp_sum(b[0]);
      if (lane == 0) A[0] = 0.f;
      __syncthreads();                 // (sc is free now: the warps' parts of B meet there and in X, A)
      if (lane == 0) dp_sm[warp] = b[0];
      __syncthreads();
      if (tid == 0) {
        float* x = rec + (3 * C + 1) * DP;
        x[0] = beta[0]; x[1] = ((dp_sm[0] + dp_sm[1]) + (dp_sm[2] + dp_sm[3])) * beta[0]; x[2] = x[3] = 0.f;
      }
      return;
    } else {
#pragma unroll
      for (int o = kSlices >> 1; o > 0; o >>= 1) {
#pragma unroll
        for (int i = 0; i < C; ++i) {
          a[i] += __shfl_xor_sync(0xffffffffu, a[i], o);
          b[i] += __shfl_xor_sync(0xffffffffu, b[i], o);
        }
      }
      if (sl == 0) {
#pragma unroll
        for (int i = 0; i < C; ++i) { A[i * C + jj] = a[i]; B[i * C + jj] = b[i]; }
      }
    }
  }
  __syncthreads();
  if (tid < C) {                       // column tid of X: forward substitution, then the row's beta
    float x[C];
#pragma unroll
    for (int i = 0; i < C; ++i) {
      float acc = 0.f;
#pragma unroll
      for (int l = 0; l < C; ++l)
        if (l < i) acc = fmaf(A[i * C + l], x[l], acc);
      x[i] = i == tid ? 1.f : (i > tid ? -beta[i] * acc : 0.f);
    }
#pragma unroll
    for (int i = 0; i < C; ++i) X[i * C + tid] = x[i] * beta[tid];
  }
  __syncthreads();
  float* xo = rec + (3 * C + 1) * DP;
  for (int x = tid; x < C * C; x += kThreads) {
    const int i = x / C, jc = x % C;
    float acc = 0.f;
#pragma unroll
    for (int l = 0; l < C; ++l) acc = fmaf(l <= i ? B[i * C + l] : 0.f, X[l * C + jc], acc);
    xo[x] = X[x];
    xo[C * C + x] = acc;
  }
}

struct DeltaArgs {
  const float* rec;                  // records of delta_chunk_prep_kernel
  const float* v;                    // [M, H V]
  float* o;                          // [M, H V]
  float* S; size_t slot_stride;      // [H, V, D] per slot: a column of the state (one value channel) is contiguous
  int H, D, V, DP;
  int vec;                           // D and the slot's columns are whole 16-byte pieces
};

// two fp32 products and sums at once
SSDK_DEVINL uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
SSDK_DEVINL uint64_t pack2(float x, float y) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
  return d;
}
SSDK_DEVINL void unpack2(uint64_t v, float* x, float* y) { asm("mov.b64 {%0, %1}, %2;" : "=f"(*x), "=f"(*y) : "l"(v)); }

constexpr int kDeltaWarps = 4;
inline __host__ __device__ int delta_cols(int LC, int NC) { return kDeltaWarps * 32 / LC * NC; }   // value columns of a CTA
inline size_t delta_scan_smem(int DP, int LC, int NC, int C) { return (size_t)2 * (delta_record(DP, C) + C * delta_cols(LC, NC)) * 4; }

// The walk over a sequence's chunks.  grid (n_seqs, H, ceil(V / delta_cols)), kDeltaWarps warps.  The columns of the state are
// independent of one another: LC neighbouring lanes share NC columns (1 or 2), lane r of them holds their key
// channels 4 (r + LC i) .. + 3, i < NQ, in registers (DP = 4 LC NQ); with two columns one load of a scaled key serves both.  Sums over D are
// thread-local packed products followed by a shuffle tree over the LC lanes; C rows' trees run together.  The next chunk's
// record arrives by cp.async under the current one's arithmetic.
template <int LC, int NQ, int NC, int C>
__global__ void __launch_bounds__(kDeltaWarps * 32, 1) delta_chunk_scan_kernel(const DeltaArgs p, const Ragged rg) {
  extern __shared__ __align__(16) float ds_sm[];
  constexpr int DP = 4 * LC * NQ, kCols = kDeltaWarps * 32 / LC * NC, kThreads = kDeltaWarps * 32, kVals = NC * C;
  constexpr int kRec = (3 * C + 1) * DP + (C > 1 ? 2 * C * C : 4), kBuf = kRec + C * kCols;
  const int s = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x, lr = tid % LC, jl = NC * (tid / LC), c0 = blockIdx.z * kCols, j = c0 + jl;
  const int D = p.D, V = p.V, HV = p.H * V, vcols = min(kCols, V - c0);
  const bool carried = rg.pos0[s] > 0;
  float* Sg = p.S + (size_t)rg.slot[s] * p.slot_stride + ((size_t)hd * V + j) * D;
  uint64_t S[NC][NQ][2];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int d = 4 * (lr + LC * i);
      const float* src = Sg + (size_t)c * D;
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (j + c < V && carried) {
        if (p.vec) {
          if (d < D) { const float4 f = *reinterpret_cast<const float4*>(src + d); x[0] = f.x; x[1] = f.y; x[2] = f.z; x[3] = f.w; }
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (d + e < D) x[e] = src[d + e];
        }
      }
      S[c][i][0] = pack2(x[0], x[1]); S[c][i][1] = pack2(x[2], x[3]);
    }
  for (int i = tid; i < 2 * kBuf; i += kThreads) ds_sm[i] = 0.f;   // value rows and columns outside the portion stay finite
  __syncthreads();
  const int r0 = rg.cu[s], r1 = rg.cu[s + 1], n_chunks = (r1 - r0 + C - 1) / C;
  const float* rec0 = p.rec + (delta_chunk_index(rg, s, 0, C) * p.H + hd) * kRec;
  auto issue = [&](int ci, float* buf) {
    const float* src = rec0 + (size_t)ci * p.H * kRec;
    for (int i = tid; i < kRec / 4; i += kThreads) cp_async16(buf + 4 * i, src + 4 * i, true);
    const int m0 = r0 + ci * C, nr = min(C, r1 - m0);
    for (int i = tid; i < C * kCols; i += kThreads) {
      const int r = i / kCols, c = i % kCols;
      if (r < nr && c < vcols) cp_async4(buf + kRec + i, p.v + (size_t)(m0 + r) * HV + hd * V + c0 + c);
    }
    cp_async_commit();
  };
  issue(0, ds_sm);
  for (int ci = 0; ci < n_chunks; ++ci) {
    if (ci + 1 < n_chunks) {
      issue(ci + 1, ds_sm + ((ci + 1) & 1) * kBuf);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* buf = ds_sm + (ci & 1) * kBuf;
    const float* Xs = buf + (3 * C + 1) * DP;
    const float* vs = buf + kRec + jl;
    // 16-byte pieces of a record row.  All pieces of a phase are requested together and ahead of the arithmetic before it (the
    // walk is bound by the latency of shared memory and of the exchanges, not by their number): kAll keeps a phase in registers
    const uint32_t at = smem_u32(buf) + 16u * lr;
    constexpr bool kAll = NQ * C <= 16;
    constexpr int kAhead = kAll ? C : (NQ <= 4 && C >= 4 ? 4 : 1);   // rows requested together
    typedef ulonglong2 Rows[kAhead][NQ];
    auto fetch = [&](int row0, Rows& k) {
#pragma unroll
      for (int i = 0; i < kAhead; ++i)
#pragma unroll
        for (int x = 0; x < NQ; ++x)
          asm volatile("ld.shared.v2.u64 {%0, %1}, [%2];" : "=l"(k[i][x].x), "=l"(k[i][x].y) : "r"(at + (uint32_t)((row0 + i) * DP + 4 * LC * x) * 4u) : "memory");
    };
    float P[C][NC], O[kVals];
    auto sums = [&](const Rows& k, int i0, auto put) {   // products of the fetched rows with the state before the chunk
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        uint64_t a[NC] = {};
#pragma unroll
        for (int x = 0; x < NQ; ++x)
#pragma unroll
          for (int c = 0; c < NC; ++c) { a[c] = fma2(S[c][x][0], k[i][x].x, a[c]); a[c] = fma2(S[c][x][1], k[i][x].y, a[c]); }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float lo, hi;
          unpack2(a[c], &lo, &hi);
          put(i0 + i, c, lo + hi);
        }
      }
    };
    auto put_p = [&](int i, int c, float v) { P[i][c] = v; };
    auto put_o = [&](int i, int c, float v) { O[NC * i + c] = v; };
    Rows kr;
    if constexpr (kAll) {
      Rows kg, qg;
      fetch(0, kg);
      fetch(2 * C, qg);
      sums(kg, 0, put_p);
      fetch(C, kr);
      sums(qg, 0, put_o);
    } else {
#pragma unroll
      for (int i0 = 0; i0 < C; i0 += kAhead) { fetch(i0, kr); sums(kr, i0, put_p); }
#pragma unroll
      for (int i0 = 0; i0 < C; i0 += kAhead) { fetch(2 * C + i0, kr); sums(kr, i0, put_o); }
      fetch(C, kr);
    }
    float xr[C][(C + 3) / 4 * 4];
#pragma unroll
    for (int i = 0; i < C; ++i)
#pragma unroll
      for (int l = 0; l <= i; l += 4) {
        const float4 f = *reinterpret_cast<const float4*>(Xs + i * C + l);
        xr[i][l] = f.x; xr[i][l + 1] = f.y; xr[i][l + 2] = f.z; xr[i][l + 3] = f.w;
      }
#pragma unroll
    for (int o = LC >> 1; o > 0; o >>= 1) {
      float t[C][NC];   // all exchanges of a step are in flight together
#pragma unroll
      for (int i = 0; i < C; ++i)
#pragma unroll
        for (int c = 0; c < NC; ++c) t[i][c] = __shfl_xor_sync(0xffffffffu, P[i][c], o);
#pragma unroll
      for (int i = 0; i < C; ++i)
#pragma unroll
        for (int c = 0; c < NC; ++c) P[i][c] += t[i][c];
    }
    float r[C][NC];
#pragma unroll
    for (int i = 0; i < C; ++i)
#pragma unroll
      for (int c = 0; c < NC; ++c) r[i][c] = vs[i * kCols + c] - P[i][c];
    // the state: decay of the whole chunk, then every row's write u_i = sum_l X_il r_l
#pragma unroll
    for (int x = 0; x < NQ; ++x) {
      const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(buf + 3 * C * DP + 4 * (lr + LC * x));
#pragma unroll
      for (int c = 0; c < NC; ++c) { S[c][x][0] = fma2(S[c][x][0], g.x, S[c][x][0]); S[c][x][1] = fma2(S[c][x][1], g.y, S[c][x][1]); }
    }
#pragma unroll
    for (int i0 = 0; i0 < C; i0 += kAhead) {
      if (i0 > 0) fetch(C + i0, kr);
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float u = 0.f;
#pragma unroll
          for (int l = 0; l <= i0 + i; ++l) u = fmaf(xr[i0 + i][l], r[l][c], u);
          const uint64_t uu = pack2(u, u);
#pragma unroll
          for (int x = 0; x < NQ; ++x) { S[c][x][0] = fma2(kr[i][x].x, uu, S[c][x][0]); S[c][x][1] = fma2(kr[i][x].y, uu, S[c][x][1]); }
        }
      }
    }
    // the read-out: the lanes' parts are summed so that a lane ends with its own value(s), index NC row + column (lanes share one
    // when there are fewer values than lanes)
    const int m0 = r0 + ci * C, nr = min(C, r1 - m0);
#pragma unroll
    for (int o = LC >> 1, n = kVals >> 1; o > 0; o >>= 1, n >>= 1) {
      const bool up = (lr & o) != 0;
      float got[kVals];
#pragma unroll
      for (int x = 0; x < kVals; ++x)
        if (x < n) got[x] = __shfl_xor_sync(0xffffffffu, up ? O[x] : O[x + n], o);
        else if (n == 0 && x == 0) got[0] = __shfl_xor_sync(0xffffffffu, O[0], o);
#pragma unroll
      for (int x = 0; x < kVals; ++x)
        if (x < n) O[x] = (up ? O[x + n] : O[x]) + got[x];
        else if (n == 0 && x == 0) O[0] += got[0];
    }
    constexpr int kEach = kVals > LC ? kVals / LC : 1, kShare = kVals < LC ? LC / kVals : 1;
#pragma unroll
    for (int x = 0; x < kEach; ++x) {
      const int idx = lr / kShare * kEach + x, i = idx / NC, c = idx % NC;
      float acc = O[x];
#pragma unroll
      for (int l = 0; l < C; ++l) acc = fmaf(Xs[(C > 1 ? C * C : 1) + i * C + l], NC == 2 && c ? r[l][NC - 1] : r[l][0], acc);
      if (lr % kShare == 0 && i < nr && j + c < V) p.o[(size_t)(m0 + i) * HV + hd * V + j + c] = acc;
    }
    __syncthreads();  // every thread is done with this buffer before the chunk after next is copied into it
  }
#pragma unroll
  for (int c = 0; c < NC; ++c)
    if (j + c < V) {
#pragma unroll
      for (int i = 0; i < NQ; ++i) {
        const int d = 4 * (lr + LC * i);
        float* dst = Sg + (size_t)c * D;
        float x[4];
        unpack2(S[c][i][0], x, x + 1); unpack2(S[c][i][1], x + 2, x + 3);
        if (p.vec) {
          if (d < D) *reinterpret_cast<float4*>(dst + d) = make_float4(x[0], x[1], x[2], x[3]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (d + e < D) dst[d + e] = x[e];
        }
      }
    }
}

// Any D: one thread per column, the column in shared memory ([D][blockDim], dynamic), records of single rows (C = 1) read from
// global memory.  grid (n_seqs, H, ceil(V / blockDim))
__global__ void delta_scan_any_kernel(const DeltaArgs p, const Ragged rg) {
  extern __shared__ __align__(16) float ds_sm[];
  const int s = blockIdx.x, hd = blockIdx.y, jl = threadIdx.x, Vr = blockDim.x, j = blockIdx.z * Vr + jl;
  const int D = p.D, V = p.V, DP = p.DP, kRec = delta_record(DP, 1);
  if (j >= V) return;
  float* Sg = p.S + (size_t)rg.slot[s] * p.slot_stride + ((size_t)hd * V + j) * D;
  const bool carried = rg.pos0[s] > 0;
  for (int d = 0; d < D; ++d) ds_sm[(size_t)d * Vr + jl] = carried ? Sg[d] : 0.f;
  for (int ci = 0; ci < rg.cu[s + 1] - rg.cu[s]; ++ci) {
    const float* rec = p.rec + (delta_chunk_index(rg, s, ci, 1) * p.H + hd) * kRec;
    const size_t at = ((size_t)(rg.cu[s] + ci) * p.H + hd) * V + j;
    float dot = 0.f, o = 0.f;
    for (int d = 0; d < D; ++d) {
      const float sv = ds_sm[(size_t)d * Vr + jl];
      dot = fmaf(sv, rec[d], dot);
      o = fmaf(sv, rec[2 * DP + d], o);
    }
    const float r = p.v[at] - dot, u = rec[4 * DP] * r;
    for (int d = 0; d < D; ++d) {
      const float sv = ds_sm[(size_t)d * Vr + jl];
      ds_sm[(size_t)d * Vr + jl] = fmaf(rec[DP + d], u, fmaf(sv, rec[3 * DP + d], sv));
    }
    p.o[at] = fmaf(rec[4 * DP + 1], r, o);
  }
  for (int d = 0; d < D; ++d) Sg[d] = ds_sm[(size_t)d * Vr + jl];
}

// fp32 columns [c0, c0 + n1) and [c0 + n1, c0 + n1 + n2) of each row -> two dense T matrices (operands of two linear layers)
template <typename T>
__global__ void cast_split_kernel(const float* __restrict__ src, int ld_src, T* __restrict__ d1, int n1, T* __restrict__ d2, int n2) {
  const float* r = src + (size_t)blockIdx.x * ld_src;
  for (int c = threadIdx.x; c < n1 + n2; c += blockDim.x) {
    if (c < n1) st_f<T>(d1 + (size_t)blockIdx.x * n1 + c, r[c]);
    else st_f<T>(d2 + (size_t)blockIdx.x * n2 + (c - n1), r[c]);
  }
}

}  // namespace ssdk
