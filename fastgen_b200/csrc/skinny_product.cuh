// The block product of the weight-streaming kernels: 16 rows of a weight matrix against a few tokens
// (see gemm_skinny.cu for the scheme).  Shared by the products of a few tokens (gemm_skinny.cu) and by
// the routed experts' (moe.cu), whose 16 rows come from two matrices and whose tokens are gathered.
#pragma once

#include "common.cuh"

namespace fg_skinny {

constexpr int ROWS = 16;   // rows of W per block
constexpr int CHUNK = 64;  // k elements per warp step
constexpr int WARPS = 8;
constexpr int THREADS = WARPS * 32;

enum { ACT_NONE = 0, ACT_GELU_ERF = 1, ACT_GELU_TANH = 2, ACT_RELU2 = 3 };

__device__ __forceinline__ float activate(float z, int act) {
  if (act == ACT_GELU_ERF) return 0.5f * z * (1.f + erff(z * 0.70710678118654752440f));
  if (act == ACT_GELU_TANH) return 0.5f * z * (1.f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
  if (act == ACT_RELU2) return z > 0.f ? z * z : 0.f;
  return z;
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// 16-byte asynchronous copy; `keep` asks for the line to stay in L1 (activations,
// read by every warp) while weights, read once, bypass it.  !pred: zero-fill.
template <bool KEEP>
__device__ __forceinline__ void cp_async_16(void* dst, const void* src, bool pred) {
  const int bytes = pred ? 16 : 0;
  if (KEEP)
    asm volatile("cp.async.ca.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes)
                 : "memory");
  else
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes)
                 : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory");
}

__device__ __forceinline__ void mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                    uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
      "{%0,%1,%2,%3};\n"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// 16-byte pieces a thread copies per chunk (4 of W, the rest of x), ring depth, ring size.
// How many blocks share an SM is chosen with the ring (up to 8 tokens; the warps' sums then go
// to the ring's memory once it is through, not to memory of their own):
//  * TWO_AN_SM: four stages, 96 KiB a block.  The shared-memory carve-out is asked to be no
//    larger than the two blocks need (196 KiB), which leaves the L1 room for x: every block reads
//    all of x, 64 KiB at 8 tokens of 4,096, and a product of 28,672 rows took 40.5 us with the
//    largest carve-out against 38.7 (36.7 with one token).
//  * THREE_AN_SM: three stages, 72 KiB.  A launch of a little more than two blocks an SM runs
//    as one round and a fraction of a second one, and the fraction costs about as much as a
//    whole round (16 rows of 4,096 a block, 8 tokens: 296 blocks 7.8 us, 320 blocks 10.7, 384
//    blocks 12.9, 592 blocks 14.7); with three blocks an SM up to 444 blocks run at once, with
//    as many bytes in flight an SM (320 blocks 9.0 us, 384 blocks 9.7).
//  * ONE_AN_SM: six stages, 144 KiB, for a launch of no more blocks than SMs: every block has
//    an SM of its own then, and half as many bytes again in flight (2,048 rows of 8,192, 8
//    tokens: 10.0 -> 7.2 us; 2,048 rows of 4,096: 5.7 -> 4.4).
enum { TWO_AN_SM = 0, THREE_AN_SM = 1, ONE_AN_SM = 2 };

template <int NT, int MODE = TWO_AN_SM>
struct Ring {
  static_assert(MODE == TWO_AN_SM || NT == 1, "the other rings are for up to 8 tokens");
  static constexpr int PIECES = 4 + 2 * NT;
  static constexpr int STAGES =
      MODE == THREE_AN_SM ? 3 : (MODE == ONE_AN_SM ? 6 : (NT == 1 ? 4 : (NT == 2 ? 3 : 2)));  // 96 KiB: two blocks an SM
  static constexpr size_t BYTES = (size_t)STAGES * PIECES * THREADS * 16;
  static constexpr bool SUMS_IN_RING = NT == 1;
  // per cent of the largest carve-out to ask for (0: the driver's choice)
  static constexpr int CARVEOUT = NT != 1 ? 0 : (MODE == THREE_AN_SM ? 100 : (MODE == ONE_AN_SM ? 70 : 80));
};

// One block's product: 16 rows of W (from row n0) against the tokens' x.  The pieces a
// thread streams, its ring and its accumulators; the callers decide when the weights'
// first stages are issued (they may go ahead of data that is not ready yet).
template <int NT, int MODE = TWO_AN_SM>
struct BlockProduct {
  static constexpr int PIECES = Ring<NT, MODE>::PIECES;
  static constexpr int STAGES = Ring<NT, MODE>::STAGES;
  uint4* ring;  // [STAGES][PIECES][THREADS]
  const __nv_bfloat16 *wa, *wb, *xr[NT];
  bool row_a, row_b, tok_ok[NT];
  float acc[NT][4];
  int K, my_chunks, tid, warp, r, c;

  // the thread's place in the block; the callers then point wa, wb and xr at column c * 8 of their rows
  // (and say which of those exist)
  __device__ __forceinline__ void begin(uint4* ring_, int K_) {
    ring = ring_;
    K = K_;
    tid = threadIdx.x;
    warp = tid >> 5;
    const int lane = tid & 31;
    r = lane >> 2;
    c = lane & 3;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    const int n_chunks = (K + CHUNK - 1) / CHUNK;
    my_chunks = warp < n_chunks ? (n_chunks - warp + WARPS - 1) / WARPS : 0;
  }

  __device__ __forceinline__ void setup(uint4* ring_, const __nv_bfloat16* x, int ldx, const __nv_bfloat16* w, int ldw,
                                        int M, int N, int K_, int n0) {
    begin(ring_, K_);
    // rows beyond N and tokens beyond M are zero-filled and discarded at the end
    row_a = n0 + r < N;
    row_b = n0 + r + 8 < N;
    wa = w + (size_t)(row_a ? n0 + r : 0) * ldw + c * 8;
    wb = w + (size_t)(row_b ? n0 + r + 8 : 0) * ldw + c * 8;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int tok = nt * 8 + r;
      tok_ok[nt] = tok < M;
      xr[nt] = x + (size_t)(tok_ok[nt] ? tok : 0) * ldx + c * 8;
    }
  }

  // issue the copies of this thread's i-th chunk into stage i % STAGES: the pieces of
  // W, the pieces of x, or both
  __device__ __forceinline__ void issue(int i, bool do_w, bool do_x) {
    uint4* slot = ring + (size_t)(i % STAGES) * PIECES * THREADS + tid;
    const int k = (warp + i * WARPS) * CHUNK;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int kk = k + h * 32;
      const bool ok = kk + c * 8 < K;  // K is a multiple of 8: a 16-byte piece is all in or all out
      if (do_w) {
        cp_async_16<false>(slot + (2 * h) * THREADS, wa + kk, ok && row_a);
        cp_async_16<false>(slot + (2 * h + 1) * THREADS, wb + kk, ok && row_b);
      }
      if (do_x) {
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
          cp_async_16<true>(slot + (4 + nt * 2 + h) * THREADS, xr[nt] + kk, ok && tok_ok[nt]);
      }
    }
  }

  // the weights of the first stages (they depend on nothing that is computed in the step)
  __device__ __forceinline__ void first_weights() {
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s)
      if (s < my_chunks) issue(s, true, false);
  }

  // the x pieces of the first stages, the main loop, and the warps' sums into `red`
  __device__ __forceinline__ void run(float (*red)[ROWS][NT * 8]) {
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) {
      if (s < my_chunks) issue(s, false, true);
      cp_async_commit();
    }
    for (int i = 0; i < my_chunks; ++i) {
      if (i + STAGES - 1 < my_chunks) issue(i + STAGES - 1, true, true);
      cp_async_commit();
      cp_async_wait<STAGES - 1>();  // this thread's copies of chunk i have landed; only it reads them
      const uint4* slot = ring + (size_t)(i % STAGES) * PIECES * THREADS + tid;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const uint4 a_lo = slot[(2 * h) * THREADS], a_hi = slot[(2 * h + 1) * THREADS];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const uint4 b = slot[(4 + nt * 2 + h) * THREADS];
          mma(acc[nt], a_lo.x, a_hi.x, a_lo.y, a_hi.y, b.x, b.y);
          mma(acc[nt], a_lo.z, a_hi.z, a_lo.w, a_hi.w, b.z, b.w);
        }
      }
    }
    if (Ring<NT, MODE>::SUMS_IN_RING) __syncthreads();  // `red` is the ring's memory: every thread is through with its stages
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      red[warp][r][nt * 8 + 2 * c] = acc[nt][0];
      red[warp][r][nt * 8 + 2 * c + 1] = acc[nt][1];
      red[warp][r + 8][nt * 8 + 2 * c] = acc[nt][2];
      red[warp][r + 8][nt * 8 + 2 * c + 1] = acc[nt][3];
    }
    __syncthreads();
  }
};

// the warps' partial sums of (row, token), in warp order
template <int NT>
__device__ __forceinline__ float block_total(float (*red)[ROWS][NT * 8], int row, int tok) {
  float s = 0.f;
#pragma unroll
  for (int wi = 0; wi < WARPS; ++wi) s += red[wi][row][tok];
  return s;
}

}  // namespace fg_skinny
