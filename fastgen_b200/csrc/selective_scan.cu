// The recurrence of the selective state-space mixer (Mamba-1 form): every channel c has a state of N numbers
// with a decay of its own each.  With d_c = softplus(dt_c + bias_c), in float32, token by token:
//
//   S[c, n] <- exp(d_c A[c, n]) S[c, n] + d_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c;   out_c = y_c silu(z_c)
//
// A is given times log2(e), so that the decay is one multiplication and a base-2 exponential.
//
// A block of 256 threads works on (sequence, a run of channels).  LPC neighbouring lanes share a channel, each
// with NPL consecutive numbers of its state in registers, as pairs for the packed float32 arithmetic of sm_100.
// Only S itself is a chain from token to token (one fused multiply-add a token); decays and products of the
// tokens ahead do not wait for it.  Tokens come in stages of TOK through two buffers in shared memory: the step
// sizes' softplus is taken once per (token, channel) as a stage is stored, B and C of a token are words that all
// channels of a warp share, and the next stage's numbers are on their way to registers while a stage is
// computed.  The sums over a channel's lanes are reduced for a group of tokens at a time by halving exchanges and
// pass through shared memory, so that outputs leave in runs of channels.  Tokens beyond a sequence's end have
// d = 0, which leaves the state as it is.  The recurrence runs token by token, so a prompt gives the same numbers
// however it is cut (up to the order of the sum over n, which follows the number of lanes a channel).  The state of a slot is [channels][N] float32, zero at admission.
#include "common.cuh"

constexpr int SEL_THREADS = 256;

__device__ __forceinline__ float sel_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint64_t sel_pair(float lo, float hi) {
  uint64_t v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
  return v;
}
__device__ __forceinline__ void sel_split(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t sel_mul(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t sel_fma(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ float sel_silu(float z, float*) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sel_silu(float z, __nv_bfloat16*) { return __fdividef(z, 1.f + __expf(-z)); }

// the NPL / 2 pairs at p (16-byte words where there are two pairs or more)
template <int PAIRS>
__device__ __forceinline__ void sel_pairs(const float* p, uint64_t (&v)[PAIRS]) {
  if (PAIRS == 1) {
    v[0] = *reinterpret_cast<const uint64_t*>(p);
  } else {
#pragma unroll
    for (int i = 0; i < PAIRS; i += 2) {
      const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(p + 2 * i);
      v[i] = w.x;
      v[i + 1] = w.y;
    }
  }
}

template <typename T, int LPC, int NPL, int TOK>
__global__ void __launch_bounds__(SEL_THREADS, 2)
selective_scan_kernel(const T* __restrict__ x, long x_stride, const T* __restrict__ dt, long dt_stride,
                      const T* __restrict__ z, long z_stride, const T* __restrict__ low, long low_stride, int b_offset,
                      const float* __restrict__ dt_bias, const float* __restrict__ a_log2,
                      const float* __restrict__ d_skip, T* __restrict__ out, long out_stride, float* __restrict__ state,
                      long state_stride, const int* __restrict__ seq_slot, const int* __restrict__ seq_start, int inner,
                      int N, int vec) {
  constexpr int NP = LPC * NPL;              // state numbers of a channel, padded
  constexpr int PAIRS = NPL / 2;
  constexpr int CH = SEL_THREADS / LPC;      // channels a block
  constexpr int EPT = (TOK * CH + SEL_THREADS - 1) / SEL_THREADS;
  constexpr int BPT = (TOK * NP + SEL_THREADS - 1) / SEL_THREADS;
  constexpr int GROUP = LPC < 8 ? LPC : 8;   // tokens whose sums are reduced together
  constexpr int YLD = CH + 32 / LPC;         // rows of the outputs fall on different banks
  static_assert(TOK % GROUP == 0 && NPL % 2 == 0 && SEL_THREADS % CH == 0 && LPC <= 32, "shapes of the stages");
  static_assert(PAIRS == 1 || PAIRS % 2 == 0, "pairs are read one or two at a time");
  __shared__ __align__(16) float dx_s[2][TOK][CH][4];  // d, d, d x, d x: pairs as the arithmetic takes them
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
  uint64_t S[PAIRS], a[PAIRS];
  float* st = state + (size_t)slot * state_stride + (size_t)(mine ? c0 + ch : 0) * N + sub * NPL;
  const float* ar = a_log2 + (size_t)(mine ? c0 + ch : 0) * N + sub * NPL;
  if (vec) {
    sel_pairs<PAIRS>(st, S);
    sel_pairs<PAIRS>(ar, a);
  } else {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const bool ok0 = sub * NPL + 2 * i < N, ok1 = sub * NPL + 2 * i + 1 < N;
      S[i] = sel_pair(ok0 ? st[2 * i] : 0.f, ok1 ? st[2 * i + 1] : 0.f);
      a[i] = sel_pair(ok0 ? ar[2 * i] : 0.f, ok1 ? ar[2 * i + 1] : 0.f);
    }
  }

  // loads and outputs: thread tid takes channel tid % CH of every (SEL_THREADS / CH)-th token of a stage
  const int lc = tid % CH, lt = tid / CH;
  const bool lc_ok = c0 + lc < inner;
  const float bias = lc_ok ? dt_bias[c0 + lc] : 0.f, skip = lc_ok ? d_skip[c0 + lc] : 0.f;
  // the next stage, as loaded (a conversion here would wait for the load)
  T xn[EPT], dn[EPT], zn[EPT], bn[BPT], cn[BPT];
  float xc[EPT], zc[EPT];                             // the stage at hand
  const T zero = from_f32<T>(0.f);
  constexpr int STEP = SEL_THREADS / CH;  // tokens between two elements of a thread
  const size_t row0 = (size_t)start + lt, col = lc_ok ? c0 + lc : 0;
  const T *px = x + row0 * x_stride + col, *pd = dt + row0 * dt_stride + col, *pz = z + row0 * z_stride + col;
  T* po = out + row0 * out_stride + col;
  const T* pl = low + (size_t)start * low_stride + b_offset;
  // `left`: tokens of the sequence from the stage's first on; the pointers go on to the next stage
  auto fetch = [&](int left) {
#pragma unroll
    for (int i = 0; i < EPT; ++i) {
      const int tt = lt + i * STEP;
      const bool ok = lc_ok && tt < TOK && tt < left;
      xn[i] = ok ? px[i * STEP * x_stride] : zero;
      dn[i] = ok ? pd[i * STEP * dt_stride] : zero;
      zn[i] = ok ? pz[i * STEP * z_stride] : zero;
    }
#pragma unroll
    for (int i = 0; i < BPT; ++i) {
      const int e = tid + i * SEL_THREADS, tt = e / NP, n = e % NP;
      const bool ok = tt < TOK && n < N && tt < left;
      const T* row = pl + tt * low_stride + n;
      bn[i] = ok ? row[0] : zero;
      cn[i] = ok ? row[N] : zero;
    }
    px += TOK * x_stride;
    pd += TOK * dt_stride;
    pz += TOK * z_stride;
    pl += TOK * low_stride;
  };
  auto store = [&](int buf, int left) {
#pragma unroll
    for (int i = 0; i < EPT; ++i) {
      const int tt = lt + i * STEP;
      float d = 0.f;
      if (lc_ok && tt < left) {
        const float v = to_f32<T>(dn[i]) + bias;
        d = v > 20.f ? v : log1pf(expf(v));
      }
      xc[i] = to_f32<T>(xn[i]);
      zc[i] = to_f32<T>(zn[i]);
      const float dx = d * xc[i];
      if (tt < TOK) *reinterpret_cast<float4*>(dx_s[buf][tt][lc]) = make_float4(d, d, dx, dx);
    }
#pragma unroll
    for (int i = 0; i < BPT; ++i) {
      const int e = tid + i * SEL_THREADS, tt = e / NP, n = e % NP;
      if (tt < TOK) {
        b_s[buf][tt][n] = to_f32<T>(bn[i]);
        c_s[buf][tt][n] = to_f32<T>(cn[i]);
      }
    }
  };

  const int n_stages = (n_tok + TOK - 1) / TOK;
  fetch(n_tok);
  store(0, n_tok);
  __syncthreads();
  for (int stage = 0; stage < n_stages; ++stage) {
    const int buf = stage & 1, nt = min(TOK, n_tok - stage * TOK), left = n_tok - (stage + 1) * TOK;
    if (left > 0) fetch(left);
#pragma unroll
    for (int g0 = 0; g0 < TOK; g0 += GROUP) {
      if (g0 >= nt) break;
      float acc[GROUP];
#pragma unroll
      for (int u = 0; u < GROUP; ++u) {
        const ulonglong2 dx = *reinterpret_cast<const ulonglong2*>(dx_s[buf][g0 + u][ch]);
        uint64_t b2[PAIRS], c2[PAIRS];
        sel_pairs<PAIRS>(&b_s[buf][g0 + u][sub * NPL], b2);
        sel_pairs<PAIRS>(&c_s[buf][g0 + u][sub * NPL], c2);
        uint64_t sum = 0;  // two zeros
#pragma unroll
        for (int i = 0; i < PAIRS; ++i) {
          float e0, e1;
          sel_split(sel_mul(dx.x, a[i]), e0, e1);
          S[i] = sel_fma(sel_pair(sel_ex2(e0), sel_ex2(e1)), S[i], sel_mul(dx.y, b2[i]));
          sum = i == 0 ? sel_mul(S[i], c2[i]) : sel_fma(S[i], c2[i], sum);
        }
        float s0, s1;
        sel_split(sum, s0, s1);
        acc[u] = s0 + s1;
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
      const int tt = lt + i * STEP;
      if (lc_ok && tt < nt)
        po[i * STEP * out_stride] = from_f32<T>(fmaf(skip, xc[i], y_s[tt][lc]) * sel_silu(zc[i], (T*)nullptr));
    }
    po += TOK * out_stride;
    if (left > 0) store(buf ^ 1, left);
    __syncthreads();  // the next stage is stored, and the outputs' rows are free again
  }
  if (!mine) return;
#pragma unroll
  for (int i = 0; i < PAIRS; ++i) {
    float s0, s1;
    sel_split(S[i], s0, s1);
    if (vec) {
      *reinterpret_cast<float2*>(st + 2 * i) = make_float2(s0, s1);
    } else {
      if (sub * NPL + 2 * i < N) st[2 * i] = s0;
      if (sub * NPL + 2 * i + 1 < N) st[2 * i + 1] = s1;
    }
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
  // Four numbers a lane take the fewest instructions, two the shorter time a token: two where four would leave SMs
  // without a block.  (2,048 tokens of one sequence, 2,048 channels of 16: 247 us with four, 146 us with two; 64
  // single tokens, 4,096 channels: 37 us and 65 us.)
  const long blocks4 = (long)((inner + SEL_THREADS / (N <= 16 ? 4 : 8) - 1) / (SEL_THREADS / (N <= 16 ? 4 : 8))) * n_seqs;
  if (N <= 16 && blocks4 < 148) LAUNCH(8, 2, 32);
  else if (N <= 16) LAUNCH(4, 4, 16);
  else if (N <= 32 && blocks4 < 148) LAUNCH(16, 2, 32);
  else if (N <= 32) LAUNCH(8, 4, 16);
  else if (N <= 64) LAUNCH(16, 4, 16);
  else if (N <= 128) LAUNCH(32, 4, 16);
  else LAUNCH(32, 8, 8);
#undef LAUNCH
#undef LAUNCH_T
  FG_CHECK_LAUNCH("fg_selective_scan");
  return 0;
}
