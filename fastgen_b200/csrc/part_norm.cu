// RMS norm in equal consecutive parts of a row, on a sub-layer's output on its way into the residual
// stream:
//   y[t,:]   = delta[t,:] * (rstd of its part) * w_post[:]      rstd = 1 / sqrt(mean(part^2) + eps)
//   h[t,:]   = h[t,:] + y[t,:]  (or just y)                     float32, stored back
//   out[t,:] = h[t,:], in the output's type (what the next sub-layer reads), or with w_pre the norm of
//              h[t,:] in the same parts (the model's last norm).
// Every piece is optional, so the kernel is also the plain norm (no h) and the norm of the stream (no
// delta).  One block a row; a part is summed by a fixed number of warps that depends on the number of
// parts only, so a row's result does not depend on the batch.
#include "common.cuh"

namespace {

constexpr int PN_THREADS = 256, PN_WARPS = PN_THREADS / 32;

// rstd_s[g] of the parts of kept[0 .. dim); partial: room for max(PN_WARPS, parts) floats
__device__ __forceinline__ void part_stats(const float* kept, float* partial, float* rstd_s, int parts, int size,
                                           float eps) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per = parts >= PN_WARPS ? 1 : PN_WARPS / parts;  // warps that share a part
  __syncthreads();
  for (int i = warp; i < parts * per; i += PN_WARPS) {
    const int g = i / per, j = i - g * per;
    float ss = 0.f;
    for (int d = j * 32 + lane; d < size; d += 32 * per) {
      const float v = kept[g * size + d];
      ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) partial[i] = ss;
  }
  __syncthreads();
  for (int g = threadIdx.x; g < parts; g += PN_THREADS) {
    float ss = 0.f;
    for (int j = 0; j < per; ++j) ss += partial[g * per + j];
    rstd_s[g] = 1.f / sqrtf(ss / (float)size + eps);
  }
  __syncthreads();
}

template <typename T>
__device__ __forceinline__ float4 read4(const T* p);
template <>
__device__ __forceinline__ float4 read4<float>(const float* p) {
  return *reinterpret_cast<const float4*>(p);
}
template <>
__device__ __forceinline__ float4 read4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T>
__device__ __forceinline__ void write4(T* p, float4 v);
template <>
__device__ __forceinline__ void write4<float>(float* p, float4 v) {
  *reinterpret_cast<float4*>(p) = v;
}
template <>
__device__ __forceinline__ void write4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

template <typename TD, typename TO, bool VEC>
__global__ void __launch_bounds__(PN_THREADS)
part_norm_kernel(float* h, int fresh, const TD* delta, const float* __restrict__ w_post,
                 const float* __restrict__ w_pre, TO* __restrict__ out, const int* __restrict__ rows, int dim,
                 int parts, float eps) {
  extern __shared__ __align__(16) float kept[];  // the row, between the passes
  float* rstd_s = kept + (dim + 3) / 4 * 4;
  float* partial = rstd_s + parts;
  pdl_trigger();
  const size_t base = (size_t)(rows ? rows[blockIdx.x] : blockIdx.x) * dim;
  const size_t obase = (size_t)blockIdx.x * dim;
  const int size = dim / parts;
  const bool add = h != nullptr && !fresh;
  const bool store_h = h != nullptr && rows == nullptr && delta != nullptr;
  constexpr int V = VEC ? 4 : 1;
  pdl_wait();
  if (delta != nullptr) {
    for (int d = threadIdx.x * V; d < dim; d += PN_THREADS * V) {
      if (VEC) *reinterpret_cast<float4*>(kept + d) = read4<TD>(delta + base + d);
      else kept[d] = to_f32<TD>(delta[base + d]);
    }
    part_stats(kept, partial, rstd_s, parts, size, eps);
  }
  // a thread meets the same columns in every pass, so kept[] needs no barrier between this pass and the last
  for (int d = threadIdx.x * V; d < dim; d += PN_THREADS * V) {
    if (VEC) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (add) v = *reinterpret_cast<const float4*>(h + base + d);
      if (delta != nullptr) {
        const float4 y = *reinterpret_cast<const float4*>(kept + d), w = read4<float>(w_post + d);
        const float r = rstd_s[d / size];  // (a part's size is a multiple of four here)
        v.x += y.x * r * w.x; v.y += y.y * r * w.y; v.z += y.z * r * w.z; v.w += y.w * r * w.w;
      }
      if (store_h) *reinterpret_cast<float4*>(h + base + d) = v;
      if (w_pre != nullptr) *reinterpret_cast<float4*>(kept + d) = v;
      else if (out != nullptr) write4<TO>(out + obase + d, v);
    } else {
      float v = add ? h[base + d] : 0.f;
      if (delta != nullptr) v += kept[d] * rstd_s[d / size] * w_post[d];
      if (store_h) h[base + d] = v;
      if (w_pre != nullptr) kept[d] = v;
      else if (out != nullptr) out[obase + d] = from_f32<TO>(v);
    }
  }
  if (w_pre == nullptr || out == nullptr) return;
  part_stats(kept, partial, rstd_s, parts, size, eps);
  for (int d = threadIdx.x * V; d < dim; d += PN_THREADS * V) {
    if (VEC) {
      const float4 v = *reinterpret_cast<const float4*>(kept + d), w = read4<float>(w_pre + d);
      const float r = rstd_s[d / size];
      write4<TO>(out + obase + d, make_float4(v.x * r * w.x, v.y * r * w.y, v.z * r * w.z, v.w * r * w.w));
    } else {
      out[obase + d] = from_f32<TO>(kept[d] * rstd_s[d / size] * w_pre[d]);
    }
  }
}

}  // namespace

// h: float32 [T, dim] or null; fresh: h becomes y instead of h + y.  delta: [T, dim] of delta_dtype, with
// its norm's weight w_post (float32 [dim]), or null.  w_pre: float32 [dim] or null.  out: [n_rows, dim] of
// out_dtype, or null.  rows: null, or n_rows indices into h and delta to gather (h is then left as it was).
extern "C" int fg_part_norm(float* h, int fresh, const void* delta, int delta_dtype, const float* w_post,
                            const float* w_pre, void* out, int out_dtype, const int* rows, int n_rows, int dim,
                            int parts, float eps, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  FG_CHECK_ARG(dim > 0 && parts > 0 && dim % parts == 0, "fg_part_norm: %d columns in %d equal parts", dim, parts);
  FG_CHECK_ARG(h != nullptr || delta != nullptr, "fg_part_norm: neither a stream nor a summand");
  FG_CHECK_ARG(delta == nullptr || w_post != nullptr, "fg_part_norm: a summand without its norm's weight");
  const size_t smem = sizeof(float) * ((size_t)(dim + 3) / 4 * 4 + parts + (parts > PN_WARPS ? parts : PN_WARPS));
  FG_CHECK_ARG(smem <= 48 * 1024, "fg_part_norm: a row of %d columns in %d parts does not fit shared memory", dim, parts);
  const auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = dim % 4 == 0 && (dim / parts) % 4 == 0 && aligned(h) && aligned(delta) && aligned(w_post) &&
                   aligned(w_pre) && aligned(out);
#define LAUNCH(TD, TO)                                                                                           \
  do {                                                                                                           \
    if (vec)                                                                                                     \
      fg_launch_pdl(part_norm_kernel<TD, TO, true>, dim3(n_rows), dim3(PN_THREADS), smem, stream, h, fresh,      \
                    (const TD*)delta, w_post, w_pre, (TO*)out, rows, dim, parts, eps);                           \
    else                                                                                                         \
      fg_launch_pdl(part_norm_kernel<TD, TO, false>, dim3(n_rows), dim3(PN_THREADS), smem, stream, h, fresh,     \
                    (const TD*)delta, w_post, w_pre, (TO*)out, rows, dim, parts, eps);                           \
  } while (0)
  const int key = (delta ? delta_dtype : FG_F32) * 2 + (out ? out_dtype : FG_F32);
  switch (key) {
    case 0: LAUNCH(float, float); break;
    case 1: LAUNCH(float, __nv_bfloat16); break;
    case 2: LAUNCH(__nv_bfloat16, float); break;
    case 3: LAUNCH(__nv_bfloat16, __nv_bfloat16); break;
    default: FG_CHECK_ARG(false, "fg_part_norm: bad dtypes");
  }
#undef LAUNCH
  FG_CHECK_LAUNCH("fg_part_norm");
  return 0;
}
