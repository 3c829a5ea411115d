// The two layer norms that meet between sub-layers normed on both sides, and the residual sum between them:
//
//   d = sum_i coef_i * delta_i[t, :]
//   h[t, :] += (d - mean(d)) / sqrt(var(d) + eps_c) * w_c + b_c        (float32, stored back)
//   out[t, :] = (h - mean(h)) / sqrt(var(h) + eps) * w + b
//
// The first norm closes the sub-layer before (its output may be a sum of up to four tensors that has not been
// formed yet, such as two mixers side by side), the second one opens the next sub-layer.  All arithmetic is
// float32; a variance is the mean of the squared deviations from the mean (a pass of its own over the row,
// which waits in registers).  One block a row; the order of every sum depends on dim alone.  With `rows`,
// output row i comes from input row rows[i] and h is left as it was.
#include "common.cuh"

constexpr int LNP_MAX_TERMS = 4;
constexpr int LNP_THREADS = 256;
constexpr int LNP_MAX_DIM = 4 * 8 * LNP_THREADS;

struct LnpTerms {
  const void* delta[LNP_MAX_TERMS];
  float coef[LNP_MAX_TERMS];
  int n;
};

template <typename T>
__device__ __forceinline__ float4 lnp_load4(const T* p);
template <>
__device__ __forceinline__ float4 lnp_load4<float>(const float* p) {
  const uint4 r = ld_global_16(p);
  return make_float4(__uint_as_float(r.x), __uint_as_float(r.y), __uint_as_float(r.z), __uint_as_float(r.w));
}
template <>
__device__ __forceinline__ float4 lnp_load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  uint2 r;
  asm volatile("ld.global.v2.u32 {%0,%1}, [%2];\n" : "=r"(r.x), "=r"(r.y) : "l"(p) : "memory");
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void lnp_store4(float* p, const float* v) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void lnp_store4(__nv_bfloat16* p, const float* v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 r;
  r.x = *reinterpret_cast<uint32_t*>(&a);
  r.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = r;
}

// VEC: a thread owns QUADS runs of four columns (a multiple of four columns, everything aligned), else
// 4 * QUADS columns LNP_THREADS apart.
template <typename TD, typename TO, int QUADS, bool VEC>
__global__ void __launch_bounds__(LNP_THREADS)
layer_norm_pair_kernel(float* h, LnpTerms terms, const float* __restrict__ wc, const float* __restrict__ bc,
                       float eps_c, const float* __restrict__ w, const float* __restrict__ b, float eps,
                       TO* __restrict__ out, const int* rows, int dim) {
  __shared__ float scratch[32];
  constexpr int N = 4 * QUADS;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x;
  const size_t base = (size_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * dim, obase = (size_t)blockIdx.x * dim;
  auto column = [&](int i) { return VEC ? 4 * (tid + LNP_THREADS * (i >> 2)) + (i & 3) : tid + LNP_THREADS * i; };
  // the stream is on its way while the summand is normed
  float x[N], v[N];
#pragma unroll
  for (int q = 0; q < QUADS; ++q) {
    if (VEC) {
      const int d = column(4 * q);
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d < dim) f = lnp_load4<float>(h + base + d);
      x[4 * q] = f.x; x[4 * q + 1] = f.y; x[4 * q + 2] = f.z; x[4 * q + 3] = f.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = column(4 * q + e);
        x[4 * q + e] = d < dim ? h[base + d] : 0.f;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = 0.f;
#pragma unroll
  for (int term = 0; term < LNP_MAX_TERMS; ++term) {
    if (term >= terms.n) break;
    const TD* p = static_cast<const TD*>(terms.delta[term]) + base;
    const float c = terms.coef[term];
#pragma unroll
    for (int q = 0; q < QUADS; ++q) {
      if (VEC) {
        const int d = column(4 * q);
        if (d >= dim) continue;
        const float4 f = lnp_load4<TD>(p + d);
        v[4 * q] = fmaf(c, f.x, v[4 * q]);
        v[4 * q + 1] = fmaf(c, f.y, v[4 * q + 1]);
        v[4 * q + 2] = fmaf(c, f.z, v[4 * q + 2]);
        v[4 * q + 3] = fmaf(c, f.w, v[4 * q + 3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = column(4 * q + e);
          if (d < dim) v[4 * q + e] = fmaf(c, to_f32<TD>(p[d]), v[4 * q + e]);
        }
      }
    }
  }
  // mean and 1 / sqrt(variance + e) of a row in registers (columns beyond dim hold zeros)
  auto moments = [&](const float (&r)[N], float e, float& mean, float& rstd) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) s += r[i];
    mean = block_sum(s, scratch) / (float)dim;
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const float c = column(i) < dim ? r[i] - mean : 0.f;
      sq = fmaf(c, c, sq);
    }
    rstd = 1.f / sqrtf(block_sum(sq, scratch) / (float)dim + e);
  };
  float mean, rstd;
  moments(v, eps_c, mean, rstd);
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int d = column(i);
    if (d >= dim) continue;
    x[i] += (v[i] - mean) * rstd * wc[d] + (bc != nullptr ? bc[d] : 0.f);
  }
  if (rows == nullptr) {
#pragma unroll
    for (int q = 0; q < QUADS; ++q) {
      if (VEC) {
        const int d = column(4 * q);
        if (d < dim) lnp_store4(h + base + d, x + 4 * q);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = column(4 * q + e);
          if (d < dim) h[base + d] = x[4 * q + e];
        }
      }
    }
  }
  moments(x, eps, mean, rstd);
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int d = column(i);
    if (d < dim) v[i] = (x[i] - mean) * rstd * w[d] + (b != nullptr ? b[d] : 0.f);
  }
#pragma unroll
  for (int q = 0; q < QUADS; ++q) {
    if (VEC) {
      const int d = column(4 * q);
      if (d < dim) lnp_store4(out + obase + d, v + 4 * q);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = column(4 * q + e);
        if (d < dim) out[obase + d] = from_f32<TO>(v[4 * q + e]);
      }
    }
  }
}

template <typename TD, typename TO>
static void lnp_launch(float* h, const LnpTerms& terms, const float* wc, const float* bc, float eps_c, const float* w,
                       const float* b, float eps, TO* out, const int* rows, int n_rows, int dim, bool vec,
                       cudaStream_t stream) {
#define LAUNCH(QUADS)                                                                                                 \
  do {                                                                                                                \
    if (vec)                                                                                                          \
      fg_launch_pdl(layer_norm_pair_kernel<TD, TO, QUADS, true>, dim3(n_rows), dim3(LNP_THREADS), 0, stream, h,       \
                    terms, wc, bc, eps_c, w, b, eps, out, rows, dim);                                                 \
    else                                                                                                              \
      fg_launch_pdl(layer_norm_pair_kernel<TD, TO, QUADS, false>, dim3(n_rows), dim3(LNP_THREADS), 0, stream, h,      \
                    terms, wc, bc, eps_c, w, b, eps, out, rows, dim);                                                 \
  } while (0)
  const int quads = (dim + 4 * LNP_THREADS - 1) / (4 * LNP_THREADS);
  if (quads <= 1) LAUNCH(1);
  else if (quads <= 2) LAUNCH(2);
  else if (quads <= 4) LAUNCH(4);
  else LAUNCH(8);
#undef LAUNCH
}

extern "C" int fg_layer_norm_pair_max_dim() { return LNP_MAX_DIM; }

// h: float32 [., dim].  deltas: n_terms (1 to 4) pointers to tensors of h's shape of delta_dtype, with their
// multiples.  wc, w: float32 [dim]; bc, b: float32 [dim] or null.  out: [n_rows, dim] of out_dtype.
extern "C" int fg_layer_norm_pair(float* h, const void* const* deltas, const float* coefs, int n_terms, int delta_dtype,
                                  const float* wc, const float* bc, float eps_c, const float* w, const float* b,
                                  float eps, void* out, int out_dtype, const int* rows, int n_rows, int dim,
                                  cudaStream_t stream) {
  if (n_rows == 0) return 0;
  FG_CHECK_ARG(dim > 0 && dim <= LNP_MAX_DIM, "fg_layer_norm_pair: rows of %d (at most %d)", dim, LNP_MAX_DIM);
  FG_CHECK_ARG(n_terms >= 1 && n_terms <= LNP_MAX_TERMS, "fg_layer_norm_pair: %d summands (1 to %d)", n_terms,
               LNP_MAX_TERMS);
  FG_CHECK_ARG(wc != nullptr && w != nullptr && out != nullptr, "fg_layer_norm_pair: a norm needs its weight");
  LnpTerms terms;
  terms.n = n_terms;
  bool vec = dim % 4 == 0 && ((uintptr_t)h & 15) == 0 && ((uintptr_t)out & 15) == 0;
  for (int i = 0; i < LNP_MAX_TERMS; ++i) {
    terms.delta[i] = i < n_terms ? deltas[i] : nullptr;
    terms.coef[i] = i < n_terms ? coefs[i] : 0.f;
    vec = vec && ((uintptr_t)terms.delta[i] & 15) == 0;
  }
#define ARGS(TO) h, terms, wc, bc, eps_c, w, b, eps, (TO*)out, rows, n_rows, dim, vec, stream
  switch (delta_dtype * 2 + out_dtype) {
    case 0: lnp_launch<float, float>(ARGS(float)); break;
    case 1: lnp_launch<float, __nv_bfloat16>(ARGS(__nv_bfloat16)); break;
    case 2: lnp_launch<__nv_bfloat16, float>(ARGS(float)); break;
    case 3: lnp_launch<__nv_bfloat16, __nv_bfloat16>(ARGS(__nv_bfloat16)); break;
    default: FG_CHECK_ARG(false, "fg_layer_norm_pair: bad dtypes");
  }
#undef ARGS
  FG_CHECK_LAUNCH("fg_layer_norm_pair");
  return 0;
}
