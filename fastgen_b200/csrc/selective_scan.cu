// The recurrence of the selective state-space mixer (Mamba-1 form): every channel c has a state of N numbers
// with a decay of its own each.  With d_c = softplus(dt_c + bias_c), in float32, token by token:
//
//   S[c, n] <- exp(d_c A[c, n]) S[c, n] + d_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c;   out_c = y_c silu(z_c)
//
// A is given times log2(e), so that the decay is one multiplication and a base-2 exponential.
//
// A block of 256 threads works on (sequence, a run of channels).  LPC neighbouring lanes share a channel, each
// with NPL consecutive numbers of its state in registers.  Only S itself is a chain from token to token (one
// fused multiply-add a token); decays and products of the tokens ahead do not wait for it.  Tokens come in
// stages of TOK through two buffers in shared memory: the step sizes' softplus is taken once per (token,
// channel) as a stage is stored, B and C of a token are read as 16-byte words that all channels of a warp
// share, and the next stage's numbers are on their way to registers while a stage is computed.  The sums over
// a channel's lanes are reduced for a group of tokens at a time by halving exchanges; the sums pass through
// shared memory so that outputs leave in runs of channels.  Tokens beyond a sequence's end have d = 0, which
// leaves the state as it is.  The order of every sum depends on N alone: prompt portions, single tokens and
// mixed batches give the same numbers however a prompt is cut.  The state of a slot is [channels][N] float32,
// zero at admission.
#include "common.cuh"

constexpr int SEL_THREADS = 256;

__device__ __forceinline__ float sel_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float sel_silu(float z, float*) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sel_silu(float z, __nv_bfloat16*) { return __fdividef(z, 1.f + __expf(-z)); }

template <typename T, int LPC, int NPL, int TOK>
__global__ void __launch_bounds__(SEL_THREADS)
selective_scan_kernel(const T* __restrict__ x, long x_stride, const T* __restrict__ dt, long dt_stride,
                      const T* __restrict__ z, long z_stride, const T* __restrict__ low, long low_stride, int b_offset,
                      const float* __restrict__ dt_bias, const float* __restrict__ a_log2,
                      const float* __restrict__ d_skip, T* __restrict__ out, long out_stride, float* __restrict__ state,
                      long state_stride, const int* __restrict__ seq_slot, const int* __restrict__ seq_start, int inner,
                      int N, int vec) {
  constexpr int NP = LPC * NPL;              // state numbers of a channel, padded
  constexpr int CH = SEL_THREADS / LPC;      // channels a block
  constexpr int EPT = (TOK * CH + SEL_THREADS - 1) / SEL_THREADS;
  constexpr int BPT = (TOK * NP + SEL_THREADS - 1) / SEL_THREADS;
  constexpr int GROUP = LPC < 8 ? LPC : 8;   // tokens whose sums are reduced together
  constexpr int YLD = CH + 32 / LPC;         // rows of the outputs fall on different banks
  static_assert(TOK % GROUP == 0 && NPL % 4 == 0 && SEL_THREADS % CH == 0 && LPC <= 32, "shapes of the stages");
  __shared__ float2 dx_s[2][TOK][CH];                 // (d, d x)
  __shared__ __align__(16) float b_s[2][TOK][NP], c_s[2][TOK][NP];
  __shared__ float y_s[TOK][YLD];

  const int slot = seq_slot[blockIdx.y];
  if (slot < 0) return;
  const int start = seq_start[blockIdx.y], n_tok = seq_start[blockIdx.y + 1] - start;
  if (n_tok <= 0) return;
  const int tid = threadIdx.x;
  const int sub = tid % LPC, ch = tid / LPC;
  const int c0 = blockIdx.x * CH;
  const bool mine = c0 + ch < inner;
  // this thread's numbers of its channel's state, and their decay rates
  float S[NPL], a[NPL];
  float* st = state + (size_t)slot * state_stride + (size_t)(mine ? c0 + ch : 0) * N + sub * NPL;
  const float* ar = a_log2 + (size_t)(mine ? c0 + ch : 0) * N + sub * NPL;
  if (vec) {
#pragma unroll
    for (int i = 0; i < NPL; i += 4) {
      const float4 s4 = *reinterpret_cast<const float4*>(st + i), a4 = *reinterpret_cast<const float4*>(ar + i);
      S[i] = s4.x; S[i + 1] = s4.y; S[i + 2] = s4.z; S[i + 3] = s4.w;
      a[i] = a4.x; a[i + 1] = a4.y; a[i + 2] = a4.z; a[i + 3] = a4.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
      const bool ok = sub * NPL + i < N;
      S[i] = ok ? st[i] : 0.f;
      a[i] = ok ? ar[i] : 0.f;
    }
  }

  // loads and outputs: thread tid takes channel tid % CH of every (SEL_THREADS / CH)-th token of a stage
  const int lc = tid % CH, lt = tid / CH;
  const bool lc_ok = c0 + lc < inner;
  const float bias = lc_ok ? dt_bias[c0 + lc] : 0.f, skip = lc_ok ? d_skip[c0 + lc] : 0.f;
  float xn[EPT], dn[EPT], zn[EPT], bn[BPT], cn[BPT];  // the next stage
  float xc[EPT], zc[EPT];                             // the stage at hand
  auto fetch = [&](int stage) {
    const int t0 = stage * TOK;
#pragma unroll
    for (int i = 0; i < EPT; ++i) {
      const int tt = lt + i * (SEL_THREADS / CH), t = t0 + tt;
      const bool ok = lc_ok && tt < TOK && t < n_tok;
      const size_t row = (size_t)(start + (ok ? t : 0));
      xn[i] = ok ? to_f32<T>(x[row * x_stride + c0 + lc]) : 0.f;
      dn[i] = ok ? to_f32<T>(dt[row * dt_stride + c0 + lc]) : 0.f;
      zn[i] = ok ? to_f32<T>(z[row * z_stride + c0 + lc]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < BPT; ++i) {
      const int e = tid + i * SEL_THREADS, tt = e / NP, n = e % NP, t = t0 + tt;
      const bool ok = tt < TOK && n < N && t < n_tok;
      const T* row = low + (size_t)(start + (ok ? t : 0)) * low_stride + b_offset + (ok ? n : 0);
      bn[i] = ok ? to_f32<T>(row[0]) : 0.f;
      cn[i] = ok ? to_f32<T>(row[N]) : 0.f;
    }
  };
  auto store = [&](int stage) {
    const int buf = stage & 1, t0 = stage * TOK;
#pragma unroll
    for (int i = 0; i < EPT; ++i) {
      const int tt = lt + i * (SEL_THREADS / CH);
      float d = 0.f;
      if (lc_ok && t0 + tt < n_tok) {
        const float v = dn[i] + bias;
        d = v > 20.f ? v : log1pf(expf(v));
      }
      if (tt < TOK) dx_s[buf][tt][lc] = make_float2(d, d * xn[i]);
      xc[i] = xn[i];
      zc[i] = zn[i];
    }
#pragma unroll
    for (int i = 0; i < BPT; ++i) {
      const int e = tid + i * SEL_THREADS, tt = e / NP, n = e % NP;
      if (tt < TOK) {
        b_s[buf][tt][n] = bn[i];
        c_s[buf][tt][n] = cn[i];
      }
    }
  };

  const int n_stages = (n_tok + TOK - 1) / TOK;
  fetch(0);
  store(0);
  __syncthreads();
  for (int stage = 0; stage < n_stages; ++stage) {
    const int buf = stage & 1, nt = min(TOK, n_tok - stage * TOK);
    if (stage + 1 < n_stages) fetch(stage + 1);
#pragma unroll
    for (int g0 = 0; g0 < TOK; g0 += GROUP) {
      if (g0 >= nt) break;
      float acc[GROUP];
#pragma unroll
      for (int u = 0; u < GROUP; ++u) {
        const float2 dx = dx_s[buf][g0 + u][ch];
        float a0 = 0.f, a1 = 0.f;
#pragma unroll
        for (int i = 0; i < NPL; i += 4) {
          const float4 b4 = *reinterpret_cast<const float4*>(&b_s[buf][g0 + u][sub * NPL + i]);
          const float4 c4 = *reinterpret_cast<const float4*>(&c_s[buf][g0 + u][sub * NPL + i]);
          S[i] = fmaf(sel_ex2(dx.x * a[i]), S[i], dx.y * b4.x);
          a0 = fmaf(S[i], c4.x, a0);
          S[i + 1] = fmaf(sel_ex2(dx.x * a[i + 1]), S[i + 1], dx.y * b4.y);
          a1 = fmaf(S[i + 1], c4.y, a1);
          S[i + 2] = fmaf(sel_ex2(dx.x * a[i + 2]), S[i + 2], dx.y * b4.z);
          a0 = fmaf(S[i + 2], c4.z, a0);
          S[i + 3] = fmaf(sel_ex2(dx.x * a[i + 3]), S[i + 3], dx.y * b4.w);
          a1 = fmaf(S[i + 3], c4.w, a1);
        }
        acc[u] = a0 + a1;
      }
      // halving exchanges: after the step with mask m a lane keeps the half of its sums that its bit m
      // chooses, with the partner's share added; the masks left over add what is left
      int token = 0;
#pragma unroll
      for (int half = GROUP / 2, mask = LPC / 2; half >= 1; half >>= 1, mask >>= 1) {
        const bool upper = (sub & mask) != 0;
#pragma unroll
        for (int j = 0; j < half; ++j) {
          const float send = upper ? acc[j] : acc[j + half];
          const float keep = upper ? acc[j + half] : acc[j];
          acc[j] = keep + __shfl_xor_sync(0xffffffffu, send, mask);
        }
        token += upper ? half : 0;
      }
      constexpr int REST = LPC / GROUP;
#pragma unroll
      for (int mask = REST / 2; mask >= 1; mask >>= 1) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], mask);
      if (sub % REST == 0) y_s[g0 + token][ch] = acc[0];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < EPT; ++i) {
      const int tt = lt + i * (SEL_THREADS / CH);
      if (lc_ok && tt < nt)
        out[(size_t)(start + stage * TOK + tt) * out_stride + c0 + lc] =
            from_f32<T>(fmaf(skip, xc[i], y_s[tt][lc]) * sel_silu(zc[i], (T*)nullptr));
    }
    if (stage + 1 < n_stages) store(stage + 1);
    __syncthreads();  // the next stage is stored, and the outputs' rows are free again
  }
  if (!mine) return;
  if (vec) {
#pragma unroll
    for (int i = 0; i < NPL; i += 4)
      *reinterpret_cast<float4*>(st + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < NPL; ++i)
      if (sub * NPL + i < N) st[i] = S[i];
  }
}

// x, dt, z: [T, inner] and low: B in the N columns from b_offset, C in the N behind them, all of `dtype` with
// row strides.  dt_bias, d_skip: float32 [inner]; a_log2: float32 [inner, N], A times log2(e).  out: [T, inner]
// of `dtype`.  state: float32 [slots, state_stride], a slot's first inner * N numbers.
extern "C" int fg_selective_scan(const void* x, long x_stride, const void* dt, long dt_stride, const void* z,
                                 long z_stride, const void* low, long low_stride, long b_offset, int dtype,
                                 const float* dt_bias, const float* a_log2, const float* d_skip, void* out,
                                 long out_stride, float* state, long state_stride, const int* seq_slot,
                                 const int* seq_start, int n_seqs, int inner, int N, cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  FG_CHECK_ARG(inner > 0 && N >= 1 && N <= 256, "fg_selective_scan: %d channels of %d numbers (1 to 256)", inner, N);
  FG_CHECK_ARG(n_seqs <= 65535, "fg_selective_scan: %d sequences", n_seqs);
  FG_CHECK_ARG(state_stride >= (long)inner * N, "fg_selective_scan: a state of %ld numbers is too small", state_stride);
  FG_CHECK_ARG(dtype == FG_F32 || dtype == FG_BF16, "fg_selective_scan: bad dtype %d", dtype);
#define LAUNCH_T(T, LPC, NPL, TOK)                                                                                     \
  selective_scan_kernel<T, LPC, NPL, TOK><<<dim3((inner + SEL_THREADS / LPC - 1) / (SEL_THREADS / LPC), n_seqs),       \
                                            SEL_THREADS, 0, stream>>>(                                                 \
      (const T*)x, x_stride, (const T*)dt, dt_stride, (const T*)z, z_stride, (const T*)low, low_stride, (int)b_offset, \
      dt_bias, a_log2, d_skip, (T*)out, out_stride, state, state_stride, seq_slot, seq_start, inner, N,                \
      N == LPC * NPL && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0 && ((uintptr_t)a_log2 & 15) == 0)
#define LAUNCH(LPC, NPL, TOK)                                  \
  do {                                                         \
    if (dtype == FG_F32) LAUNCH_T(float, LPC, NPL, TOK);       \
    else LAUNCH_T(__nv_bfloat16, LPC, NPL, TOK);               \
  } while (0)
  if (N <= 16) LAUNCH(4, 4, 16);
  else if (N <= 32) LAUNCH(8, 4, 16);
  else if (N <= 64) LAUNCH(16, 4, 16);
  else if (N <= 128) LAUNCH(16, 8, 8);
  else LAUNCH(32, 8, 8);
#undef LAUNCH
#undef LAUNCH_T
  FG_CHECK_LAUNCH("fg_selective_scan");
  return 0;
}
