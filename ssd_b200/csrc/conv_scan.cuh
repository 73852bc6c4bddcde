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
//   delta_prep_kernel     convolution + SiLU of q | k | v, unit vectors per head for q and k, beta and the head decay
//   delta_scan_kernel     gated delta rule: S = g S; u = beta (v - S^T k); S += k u^T; o = S^T q
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
struct DeltaPrepArgs {
  ConvArgs conv;          // over the q | k | v columns (C = 2 G D + H V); out / out_t unused
  const float* b; int ld_b;    // [M, ...]: beta pre-activations in columns [0, H)
  const float* a; int ld_a;    // decay pre-activations: [M, ...] columns [0, H), or (per_channel) [M, H D]
  const void* A_log;      // [H] T
  const void* dt_bias;    // [H] T, or (per_channel) [H D]
  float* q;               // [M, G D] unit vectors * q_scale
  float* k;               // [M, G D] unit vectors
  float* v;               // [M, H V]
  float* beta;            // [M, H]
  float* decay;           // g - 1 (exact also where the decay g is within an ulp of 1): [M, H], or (per_channel) [M, H D]; may be `a` itself
  int H, G, D, V, per_channel;
  float q_scale, unit_eps;
};

// grid (M, 2 G + H (+ H when per_channel)): unit u < G is a query head, u < 2 G a key head, then value heads, then the decays of
// the heads' key channels; one CTA convolves the unit's channels (SiLU), and makes a query or key head a unit vector.
// dynamic shared memory: max(D, V) floats.
template <typename T>
__global__ void delta_prep_kernel(const DeltaPrepArgs p, const Ragged rg) {
  extern __shared__ float dp_sm[];
  __shared__ float red[33];
  const int m = blockIdx.x, unit = blockIdx.y, s = rg.tok_seq[m], t = m - rg.cu[s];
  const int GD = p.G * p.D, HV = p.H * p.V;
  if (unit == 0) {
    for (int h = threadIdx.x; h < p.H; h += blockDim.x) {
      p.beta[(size_t)m * p.H + h] = sigmoid_f(p.b[(size_t)m * p.ld_b + h]);
      if (!p.per_channel) {
        const float sp = softplus_f(p.a[(size_t)m * p.ld_a + h] + ld_f<T>((const T*)p.dt_bias + h));
        p.decay[(size_t)m * p.H + h] = expm1f(-expf(ld_f<T>((const T*)p.A_log + h)) * sp);
      }
    }
  }
  if (unit >= 2 * p.G + p.H) {  // the decays of one head's key channels
    const int h = unit - 2 * p.G - p.H;
    const float rate = -expf(ld_f<T>((const T*)p.A_log + h));
    for (int d = threadIdx.x; d < p.D; d += blockDim.x) {
      const int c = h * p.D + d;
      p.decay[(size_t)m * p.H * p.D + c] = expm1f(rate * softplus_f(p.a[(size_t)m * p.ld_a + c] + ld_f<T>((const T*)p.dt_bias + c)));
    }
    return;
  }
  if (unit >= 2 * p.G) {  // a value head: convolution and SiLU only
    const int c0 = 2 * GD + (unit - 2 * p.G) * p.V;
    for (int d = threadIdx.x; d < p.V; d += blockDim.x)
      p.v[(size_t)m * HV + (size_t)(unit - 2 * p.G) * p.V + d] = silu_f(conv_at<T>(p.conv, rg, m, s, t, c0 + d));
    return;
  }
  const int c0 = unit * p.D;  // q heads, then k heads, in the order of the convolution's channels
  float ss = 0.f;
  for (int d = threadIdx.x; d < p.D; d += blockDim.x) {
    const float v = silu_f(conv_at<T>(p.conv, rg, m, s, t, c0 + d));
    dp_sm[d] = v;
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const bool is_q = unit < p.G;
  const float inv = (is_q ? p.q_scale : 1.0f) / sqrtf(ss + p.unit_eps);
  float* dst = (is_q ? p.q : p.k) + (size_t)m * GD + (size_t)(is_q ? unit : unit - p.G) * p.D;
  for (int d = threadIdx.x; d < p.D; d += blockDim.x) dst[d] = dp_sm[d] * inv;
}

struct DeltaArgs {
  const float* q; const float* k;    // [M, G D]
  const float* v;                    // [M, H V]
  const float* beta;                 // [M, H]
  const float* decay;                // g - 1: [M, H], or one per key channel [M, H D]
  float* o;                          // [M, H V]
  float* S; size_t slot_stride;      // [H, V, D] per slot: a column of the state (one value channel) is contiguous
  int H, G, D, V;
  int vec;                           // D, V, row offsets and the slot are whole 16-byte pieces
};

constexpr int kDeltaRows = 16;   // rows staged together (two such buffers: the next chunk arrives under the current one's walk)
constexpr int kDeltaWarps = 4;

// floats of one staged row: k | q (| decay per channel), DP entries each, then value columns, beta, decay per head (padded to 4)
inline __host__ __device__ int delta_row_floats(int DP, int cols, bool per_channel) {
  return (per_channel ? 3 : 2) * DP + (cols + 2 + 3) / 4 * 4;
}
inline size_t delta_scan_smem(int DP, int cols, bool per_channel) {
  return (size_t)2 * kDeltaRows * delta_row_floats(DP, cols, per_channel) * 4;
}

// The walk over a sequence's rows.  grid (n_seqs, H, ceil(V / cols)), kDeltaWarps warps, cols = kDeltaWarps * 32 / LC.
// The columns of the state (value channels) are independent of one another: LC neighbouring lanes share one column, lane r
// of them holds the key channels 4 (r + LC i) .. + 3, i < NQ, in registers (D <= 4 LC NQ; padded channels meet k = q = 0).
// Both contractions over D (S^T k and S^T q) are thread-local sums followed by a shuffle tree over the LC lanes: no CTA
// barrier inside a row.  Rows arrive by cp.async, sixteen at a time, under the walk of the previous sixteen.  CH: one decay
// per key channel instead of one per head.  Everything is fp32 whatever the model's storage type.
template <int LC, int NQ, bool CH>
__global__ void __launch_bounds__(kDeltaWarps * 32) delta_scan_kernel(const DeltaArgs p, const Ragged rg) {
  extern __shared__ __align__(16) float ds_sm[];
  constexpr int DP = 4 * LC * NQ, kCols = kDeltaWarps * 32 / LC, kR = kDeltaRows, kThreads = kDeltaWarps * 32;
  const int RF = delta_row_floats(DP, kCols, CH), off_v = (CH ? 3 : 2) * DP, off_b = off_v + kCols;
  const int s = blockIdx.x, hd = blockIdx.y, g = hd / (p.H / p.G), tid = threadIdx.x;
  const int lr = tid % LC, jl = tid / LC, j = blockIdx.z * kCols + jl;
  const int D = p.D, V = p.V, GD = p.G * D, HV = p.H * V, HDk = p.H * D;
  const bool col = j < V, carried = rg.pos0[s] > 0;
  float* Sg = p.S + (size_t)rg.slot[s] * p.slot_stride + ((size_t)hd * V + (col ? j : 0)) * D;
  float4 S[NQ];
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int d = 4 * (lr + LC * i);
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (col && carried) {
      if (p.vec) {
        if (d < D) S[i] = *reinterpret_cast<const float4*>(Sg + d);
      } else {
        if (d < D) S[i].x = Sg[d];
        if (d + 1 < D) S[i].y = Sg[d + 1];
        if (d + 2 < D) S[i].z = Sg[d + 2];
        if (d + 3 < D) S[i].w = Sg[d + 3];
      }
    }
  }
  // padding (channels from D up to DP, value columns beyond V) is zero in both buffers and never written again
  for (int i = tid; i < 2 * kR * RF; i += kThreads) ds_sm[i] = 0.f;
  __syncthreads();
  const int r0 = rg.cu[s], r1 = rg.cu[s + 1];
  const int c0 = blockIdx.z * kCols, vcols = min(kCols, V - c0);
  auto issue = [&](int m0, float* buf) {
    const int nr = min(kR, r1 - m0);
    if (p.vec) {
      const int dq = D >> 2, per = (CH ? 3 : 2) * dq, vq = vcols >> 2;
      for (int i = tid; i < nr * per; i += kThreads) {
        const int r = i / per, x = i - r * per, part = x / dq, d = (x - part * dq) * 4;
        const size_t m = m0 + r;
        const float* src = part == 0 ? p.k + m * GD + g * D + d : part == 1 ? p.q + m * GD + g * D + d : p.decay + m * HDk + hd * D + d;
        cp_async16(buf + r * RF + part * DP + d, src, true);
      }
      for (int i = tid; i < nr * vq; i += kThreads) {
        const int r = i / vq, c = (i - r * vq) * 4;
        cp_async16(buf + r * RF + off_v + c, p.v + (size_t)(m0 + r) * HV + hd * V + c0 + c, true);
      }
    } else {   // 4-byte copies: no alignment rule beyond the element's own
      for (int i = tid; i < nr * D; i += kThreads) {
        const int r = i / D, d = i - r * D;
        const size_t m = m0 + r;
        cp_async4(buf + r * RF + d, p.k + m * GD + g * D + d);
        cp_async4(buf + r * RF + DP + d, p.q + m * GD + g * D + d);
        if (CH) cp_async4(buf + r * RF + 2 * DP + d, p.decay + m * HDk + hd * D + d);
      }
      for (int i = tid; i < nr * vcols; i += kThreads) {
        const int r = i / vcols, c = i - r * vcols;
        cp_async4(buf + r * RF + off_v + c, p.v + (size_t)(m0 + r) * HV + hd * V + c0 + c);
      }
    }
    if (tid < nr) {
      cp_async4(buf + tid * RF + off_b, p.beta + (size_t)(m0 + tid) * p.H + hd);
      if (!CH) cp_async4(buf + tid * RF + off_b + 1, p.decay + (size_t)(m0 + tid) * p.H + hd);
    }
    cp_async_commit();
  };
  issue(r0, ds_sm);
  int cur = 0;
  for (int m0 = r0; m0 < r1; m0 += kR, cur ^= 1) {
    const int nr = min(kR, r1 - m0);
    if (m0 + kR < r1) {
      issue(m0 + kR, ds_sm + (cur ^ 1) * kR * RF);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* buf = ds_sm + cur * kR * RF;
#pragma unroll 2
    for (int r = 0; r < nr; ++r) {
      const float* row = buf + r * RF;
      const float4* k4 = reinterpret_cast<const float4*>(row) + lr;
      const float beta = row[off_b], v = row[off_v + jl];
      float dec = 0.f;
      if (!CH) dec = row[off_b + 1];
      float4 kk[NQ];
      float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
      for (int i = 0; i < NQ; ++i) {
        kk[i] = k4[LC * i];
        const float4 gg = CH ? k4[DP / 2 + LC * i] : make_float4(dec, dec, dec, dec);
        S[i].x = fmaf(S[i].x, gg.x, S[i].x); S[i].y = fmaf(S[i].y, gg.y, S[i].y);   // S g = S + S (g - 1), rounded once
        S[i].z = fmaf(S[i].z, gg.z, S[i].z); S[i].w = fmaf(S[i].w, gg.w, S[i].w);
        a0 = fmaf(S[i].x, kk[i].x, a0); a1 = fmaf(S[i].y, kk[i].y, a1);
        a2 = fmaf(S[i].z, kk[i].z, a2); a3 = fmaf(S[i].w, kk[i].w, a3);
      }
      float dot = (a0 + a1) + (a2 + a3);
#pragma unroll
      for (int o = LC >> 1; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
      const float u = beta * (v - dot);
      a0 = a1 = a2 = a3 = 0.f;
#pragma unroll
      for (int i = 0; i < NQ; ++i) {
        const float4 qq = k4[DP / 4 + LC * i];
        S[i].x = fmaf(kk[i].x, u, S[i].x); S[i].y = fmaf(kk[i].y, u, S[i].y);
        S[i].z = fmaf(kk[i].z, u, S[i].z); S[i].w = fmaf(kk[i].w, u, S[i].w);
        a0 = fmaf(S[i].x, qq.x, a0); a1 = fmaf(S[i].y, qq.y, a1);
        a2 = fmaf(S[i].z, qq.z, a2); a3 = fmaf(S[i].w, qq.w, a3);
      }
      float o = (a0 + a1) + (a2 + a3);
#pragma unroll
      for (int x = LC >> 1; x > 0; x >>= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
      if (col && lr == 0) p.o[(size_t)(m0 + r) * HV + hd * V + j] = o;
    }
    __syncthreads();  // every thread is done with this buffer before the chunk after next is copied into it
  }
  if (col) {
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int d = 4 * (lr + LC * i);
      if (p.vec) {
        if (d < D) *reinterpret_cast<float4*>(Sg + d) = S[i];
      } else {
        if (d < D) Sg[d] = S[i].x;
        if (d + 1 < D) Sg[d + 1] = S[i].y;
        if (d + 2 < D) Sg[d + 2] = S[i].z;
        if (d + 3 < D) Sg[d + 3] = S[i].w;
      }
    }
  }
}

// Any D: one thread per column, the column in shared memory ([D][blockDim], dynamic), operands read from global memory.
// grid (n_seqs, H, ceil(V / blockDim))
template <bool CH>
__global__ void delta_scan_any_kernel(const DeltaArgs p, const Ragged rg) {
  extern __shared__ __align__(16) float ds_sm[];
  const int s = blockIdx.x, hd = blockIdx.y, g = hd / (p.H / p.G), jl = threadIdx.x, Vr = blockDim.x, j = blockIdx.z * Vr + jl;
  const int D = p.D, V = p.V;
  if (j >= V) return;
  float* Sg = p.S + (size_t)rg.slot[s] * p.slot_stride + ((size_t)hd * V + j) * D;
  const bool carried = rg.pos0[s] > 0;
  for (int d = 0; d < D; ++d) ds_sm[(size_t)d * Vr + jl] = carried ? Sg[d] : 0.f;
  for (int m = rg.cu[s]; m < rg.cu[s + 1]; ++m) {
    const float* k = p.k + (size_t)m * p.G * D + g * D;
    const float* q = p.q + (size_t)m * p.G * D + g * D;
    const float* gc = p.decay + (CH ? ((size_t)m * p.H + hd) * D : (size_t)m * p.H + hd);
    float dot = 0.f, o = 0.f;
    for (int d = 0; d < D; ++d) {
      const float so = ds_sm[(size_t)d * Vr + jl], sv = fmaf(so, gc[CH ? d : 0], so);
      ds_sm[(size_t)d * Vr + jl] = sv;
      dot = fmaf(sv, k[d], dot);
    }
    const float u = p.beta[(size_t)m * p.H + hd] * (p.v[((size_t)m * p.H + hd) * V + j] - dot);
    for (int d = 0; d < D; ++d) {
      const float sv = fmaf(k[d], u, ds_sm[(size_t)d * Vr + jl]);
      ds_sm[(size_t)d * Vr + jl] = sv;
      o = fmaf(sv, q[d], o);
    }
    p.o[((size_t)m * p.H + hd) * V + j] = o;
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
