// Attention over a cached latent for prompt portions on the 5th-generation tensor cores (bfloat16),
// compiled per latent size beside latent_mma.cu: -DFG_LATENT_RANK=R -DFG_LATENT_ROT=r.
//
// The computation of latent.cu: H query heads attend to ONE entry [c (R) | k_t (r)] per cached token; the
// score is (qa_h . c + qt_h . k_t) * scale, the output the softmax-weighted sum of the c, times
// sigmoid(gate) when a gate is given.  A block owns 128 (token, head) rows and walks the request's entries
// in tiles:
//
//   load warp:       TMA(entries of tile t) into a ring of stages, as soon as the tile that had the stage
//                    is through
//   MMA warp:        S_{t+1} = Q K_{t+1}^T (tcgen05.mma, operands in shared memory, K = all R + r columns)
//   4 softmax warps: S_t from tensor memory, one row a thread, P_t (bf16) back over S_t's columns
//   MMA warp:        O += P_t C_t (A from tensor memory; C_t is the first R columns of the same tile, read
//                    as an operand with its columns contiguous), O in tensor memory
//
// A tile in shared memory is both products' operand: it is loaded once.  The warps meet at mbarriers only,
// whose waits are bounded; the running maximum is raised, and O rescaled, only where a row's maximum grew
// by more than 2^8 (as in attention_tcgen05.cuh, whose softmax this is).
//
// With latents above 256 numbers a block owns half of the output columns (O would fill tensor memory
// otherwise) and computes all scores; entries too wide for two stages of 64 come in tiles of 32.
#include "attention_tcgen05.cuh"

#ifndef FG_LATENT_RANK
#error "compile with -DFG_LATENT_RANK and -DFG_LATENT_ROT"
#endif

namespace fg_latent_tc5 {
using namespace fg_mma;
using fg_tma::swz;
using fg_tma::tma_load_5d;

constexpr int R = FG_LATENT_RANK, ROT = FG_LATENT_ROT, D = R + ROT;
constexpr int GROUPS = (D + 63) / 64;      // 64-column groups of a tile (TMA fills columns beyond E with zeros)
constexpr int NSPLIT = R <= 256 ? 1 : 2;   // blocks that share a tile's output columns
constexpr int ROWS = 128;
constexpr int WIDTH = GROUPS * 128;        // bytes of a row over all groups
constexpr int SMEM_MAX = 220 * 1024;
constexpr int KEYS = ROWS * WIDTH + 2 * 64 * WIDTH <= SMEM_MAX ? 64 : 32;
constexpr int STAGES = ROWS * WIDTH + 3 * KEYS * WIDTH <= SMEM_MAX ? 3 : 2;
// (whole groups of output columns: R a multiple of 64, of 128 where two blocks share them)
constexpr bool SUPPORTED = R % (64 * NSPLIT) == 0 && R <= 512 && ROWS * WIDTH + STAGES * KEYS * WIDTH <= SMEM_MAX;

}  // namespace fg_latent_tc5

// 0: latents of this size are left to latent_mma.cu
extern "C" int fg_latent_tc5_rows() { return fg_latent_tc5::SUPPORTED ? fg_latent_tc5::ROWS : 0; }
extern "C" int fg_latent_tc5_keys() { return fg_latent_tc5::KEYS; }
extern "C" int fg_latent_tc5_blocks_a_tile() { return fg_latent_tc5::NSPLIT; }

#if FG_LATENT_RANK % 64 == 0 && FG_LATENT_RANK <= 512

namespace fg_latent_tc5 {
using namespace fg_tc5;  // (this namespace's own sizes hide those of the prompt kernel)

constexpr int TILE_ROWS = fg_latent_tc5::ROWS, TILE_KEYS = fg_latent_tc5::KEYS;
constexpr int E = (D + 7) / 8 * 8;         // numbers of a cache entry
constexpr int KSTEPS = (D + 15) / 16;      // instructions of a score product
constexpr int RO = R / NSPLIT;             // output columns of a block
constexpr int Q_GROUP = TILE_ROWS * 128;   // bytes of one 64-column group of the queries
constexpr int K_GROUP = TILE_KEYS * 128;   // ... of a tile
constexpr int STAGE_BYTES = GROUPS * K_GROUP;
constexpr int N_SOFTMAX = 128;
constexpr int N_THREADS = 192;             // 4 softmax warps, a load warp, an MMA warp
constexpr int LOADER = 4, ISSUER = 5;
constexpr int COL_S = 0, COL_O = 2 * TILE_KEYS;
constexpr int COLS = COL_O + RO;
constexpr int TMEM = COLS <= 64 ? 64 : COLS <= 128 ? 128 : COLS <= 256 ? 256 : 512;
constexpr size_t SMEM = (size_t)GROUPS * Q_GROUP + (size_t)STAGES * STAGE_BYTES + 1024;

__device__ __forceinline__ void tmem_st16_raw(uint32_t taddr, const uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};\n" ::"r"(taddr),
      "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]),
      "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15])
      : "memory");
  asm volatile("tcgen05.wait::st.sync.aligned;\n" ::: "memory");
}
__device__ __forceinline__ void scores_ld(uint32_t a, float (&v)[64]) { tmem_ld64(a, v); }
__device__ __forceinline__ void scores_ld(uint32_t a, float (&v)[32]) { tmem_ld32(a, v); }
__device__ __forceinline__ void probs_st(uint32_t a, const uint32_t (&v)[32]) { tmem_st32_raw(a, v); }
__device__ __forceinline__ void probs_st(uint32_t a, const uint32_t (&v)[16]) { tmem_st16_raw(a, v); }

__global__ void __launch_bounds__(N_THREADS, 1)
latent_attention_tc5_kernel(const __grid_constant__ CUtensorMap map, const __nv_bfloat16* __restrict__ qa, long qa_ts,
                            long qa_hs, const __nv_bfloat16* __restrict__ qt, long qt_ts, long qt_hs, int qt_vec,
                            __nv_bfloat16* __restrict__ out, long out_ts, long out_hs,
                            const __nv_bfloat16* __restrict__ gate, long gate_ts, const int* __restrict__ block_table,
                            int table_width, int page_size, int n_pages, const int* __restrict__ pos,
                            const int* __restrict__ tile_req, const int* __restrict__ tile_tok0,
                            const int* __restrict__ tile_ntok, int n_tiles_total, int n_heads, int heads_per_block,
                            float scale_log2, int* status) {
  extern __shared__ unsigned char smem_unaligned[];
  unsigned char* smem = reinterpret_cast<unsigned char*>(((uintptr_t)smem_unaligned + 1023) & ~(uintptr_t)1023);
  unsigned char* Qs = smem;                      // [GROUPS][128 rows][128 B]
  unsigned char* Ks = smem + GROUPS * Q_GROUP;   // [STAGES][GROUPS][keys][128 B]
  // full: a tile's entries have landed; s_done: its scores are in tensor memory; p_ready: all softmax
  // threads stored its probabilities; o_done: its P C is done (and with it every reader of its stage)
  __shared__ __align__(8) uint64_t full[STAGES], o_done[STAGES], s_done[2], p_ready[2], drained;
  __shared__ uint32_t tmem_base_s;
  __shared__ int gave_up;  // set by a wait that ran out: the waits after it return at once (see mbar_wait)

  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // the tiles are in ascending order of work and are handed out from the list's end
  const int slices = (n_heads + heads_per_block - 1) / heads_per_block * NSPLIT;
  const int tile = n_tiles_total - 1 - (int)blockIdx.x / slices;
  const int slice = (int)blockIdx.x % slices, sub = slice / NSPLIT, half = slice % NSPLIT;
  const int b = tile_req[tile], tok0 = tile_tok0[tile], ntok = tile_ntok[tile];
  auto row_token = [&](int r) { return r / heads_per_block; };
  auto row_head = [&](int r) { return sub * heads_per_block + r % heads_per_block; };
  auto row_valid = [&](int r) { return row_token(r) < ntok && row_head(r) < n_heads; };
  auto out_row = [&](int r) {
    return out + (size_t)(tok0 + row_token(r)) * out_ts + (size_t)row_head(r) * out_hs + half * RO;
  };

  if (b < 0) {
    // a tile of no request (padding of a captured step): its rows, if it names any, are zeroed
    for (int i = tid; i < TILE_ROWS * (RO / 8); i += N_THREADS) {
      const int r = i / (RO / 8), c = i - r * (RO / 8);
      if (row_valid(r)) *reinterpret_cast<uint4*>(out_row(r) + c * 8) = make_uint4(0u, 0u, 0u, 0u);
    }
    return;
  }
  if (warp == LOADER) {
    tmem_alloc(&tmem_base_s, TMEM);
    tmem_relinquish();
  }
  if (tid == N_SOFTMAX) {
    gave_up = 0;
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&o_done[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_done[i], 1);
      mbar_init(&p_ready[i], N_SOFTMAX);
    }
    mbar_init(&drained, 1);
    mbar_fence_init();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_base_s;
  const int k_end = pos[tok0] + ntok;  // tokens of a tile are consecutive positions
  const int n_tiles = (k_end + TILE_KEYS - 1) / TILE_KEYS;

  if (warp == LOADER) {
    // ================================ load warp ================================
    const int* table_row = block_table + (size_t)b * table_width;
    const int box_rows = min(page_size, TILE_KEYS);
    const int n_boxes = TILE_KEYS / box_rows;
    // the page of this lane's box of tile t (-1: no position of the request in it)
    auto look = [&](int t) {
      int page = -1;
      const int j0 = t * TILE_KEYS + lane * box_rows;
      if (lane < n_boxes && j0 < k_end) {
        const int logical = j0 / page_size;
        page = logical < table_width ? table_row[logical] : -1;
        if (page < 0 || page >= n_pages) {
          if (status) atomicOr(status, FG_STATUS_BAD_PAGE);
          page = -1;
        }
      }
      return page;
    };
    int page = look(0), stage = 0, parity = 0;
    for (int t = 0; t < n_tiles; ++t) {
      const int next = look(t + 1);  // on its way while this tile's stage becomes free
      if (t >= STAGES) mbar_wait(&o_done[stage], parity ^ 1, status, &gave_up);
      unsigned char* dst = Ks + stage * STAGE_BYTES;
      const unsigned valid = __ballot_sync(0xffffffffu, page >= 0);
      if (__popc(valid) < n_boxes) {
        // boxes without a position hold zeros (a masked probability times garbage could be NaN)
        for (int i = 0; i < n_boxes; ++i) {
          if (valid >> i & 1) continue;
          for (int g = 0; g < GROUPS; ++g)
            for (int c = lane; c < box_rows * 8; c += 32)
              *reinterpret_cast<uint4*>(dst + g * K_GROUP + i * box_rows * 128 + c * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
        fence_async_smem();
      }
      __syncwarp();
      if (lane == 0) mbar_arrive_expect(&full[stage], __popc(valid) * box_rows * WIDTH);
      for (int i = 0; i < n_boxes; ++i) {
        const int p = __shfl_sync(0xffffffffu, page, i);
        if (lane == 0 && p >= 0) {
          const int slot = (t * TILE_KEYS + i * box_rows) & (page_size - 1);
#pragma unroll
          for (int g = 0; g < GROUPS; ++g)
            tma_load_5d(dst + g * K_GROUP + i * box_rows * 128, &map, g * 64, slot, 0, p, 0, &full[stage]);
        }
      }
      page = next;
      if (++stage == STAGES) {
        stage = 0;
        parity ^= 1;
      }
    }
  } else {
    // the other warps bring the queries into the K-major operand layout (16-byte pieces, swizzled); rows
    // without a query and columns from D on hold zeros
    constexpr int PIECES = KSTEPS * 2;
    const int first = warp == ISSUER ? tid - 32 : tid;  // 160 threads, without the load warp
#pragma unroll 4
    for (int i = first; i < TILE_ROWS * PIECES; i += N_THREADS - 32) {
      const int r = i / PIECES, c = i - r * PIECES;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (row_valid(r)) {
        const size_t tk = tok0 + row_token(r), hh = row_head(r);
        if (c < R / 8) {
          v = *reinterpret_cast<const uint4*>(qa + tk * qa_ts + hh * qa_hs + c * 8);
        } else {
          const __nv_bfloat16* src = qt + tk * qt_ts + hh * qt_hs;
          const int d0 = c * 8 - R;
          if (qt_vec && d0 + 8 <= ROT) {
            v = *reinterpret_cast<const uint4*>(src + d0);
          } else {
            __nv_bfloat16* e = reinterpret_cast<__nv_bfloat16*>(&v);
#pragma unroll
            for (int k = 0; k < 8; ++k)
              if (d0 + k < ROT) e[k] = src[d0 + k];
          }
        }
      }
      *reinterpret_cast<uint4*>(Qs + (c / 8) * Q_GROUP + swz(r, c % 8)) = v;
    }
    fence_async_smem();  // written by ordinary stores, read by the tensor core
    asm volatile("bar.sync 1, %0;\n" ::"n"(N_THREADS - 32) : "memory");

    if (warp == ISSUER) {
      // ================================ MMA warp ================================
      // One thread issues everything; products run in the order of issue, so the S that overwrites the
      // columns of the S / P two tiles back follows that tile's P C by itself.
      if (lane == 0) {
        constexpr uint32_t IDESC_S = instr_desc(TILE_KEYS, false), IDESC_O = instr_desc(RO, true);
        const uint64_t q_desc = smem_desc(Qs, 16), k_desc = smem_desc(Ks, 16);
        const uint64_t c_desc = smem_desc(Ks + half * (RO / 64) * K_GROUP, K_GROUP);
        int s_stage = 0, s_parity = 0;
        auto issue_s = [&](int t) {
          mbar_wait(&full[s_stage], s_parity, status, &gave_up);
          tc_fence_after();
          const uint64_t kd = k_desc + (uint64_t)((s_stage * STAGE_BYTES) >> 4);
#pragma unroll
          for (int kk = 0; kk < KSTEPS; ++kk)
            umma_f16(tmem + COL_S + (t & 1) * TILE_KEYS, q_desc + (uint64_t)(((kk / 4) * Q_GROUP + (kk % 4) * 32) >> 4),
                     kd + (uint64_t)(((kk / 4) * K_GROUP + (kk % 4) * 32) >> 4), IDESC_S, kk > 0 ? 1u : 0u);
          umma_commit(&s_done[t & 1]);
          if (++s_stage == STAGES) {
            s_stage = 0;
            s_parity ^= 1;
          }
        };
        issue_s(0);
        int o_stage = 0;
        for (int t = 0; t < n_tiles; ++t) {
          if (t + 1 < n_tiles) issue_s(t + 1);
          // all softmax threads have stored P_t (and rescaled O where needed)
          mbar_wait(&p_ready[t & 1], (t >> 1) & 1, status, &gave_up);
          tc_fence_after();
          const uint64_t cd = c_desc + (uint64_t)((o_stage * STAGE_BYTES) >> 4);
#pragma unroll
          for (int j = 0; j < TILE_KEYS / 16; ++j)
            umma_f16_ts(tmem + COL_O, tmem + COL_S + (t & 1) * TILE_KEYS + j * 8, cd + (uint64_t)((j * 16 * 128) >> 4),
                        IDESC_O, (t > 0 || j > 0) ? 1u : 0u);
          umma_commit(&o_done[o_stage]);
          if (++o_stage == STAGES) o_stage = 0;
        }
      }
      __syncwarp();
    } else {
      // =============================== softmax warps ===============================
      const uint32_t my_lane = (uint32_t)(warp * 32) << 16;  // this warp's quarter of the TMEM lanes
      const bool my_valid = row_valid(tid);
      const int my_pos = my_valid ? pos[tok0 + row_token(tid)] : -1;
      float m_ref = -INFINITY, l_run = 0.f;
      const float c = scale_log2;
      const bool warp_full = __all_sync(0xffffffffu, my_valid);
      int warp_min = my_valid ? my_pos : 0x7fffffff;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) warp_min = min(warp_min, __shfl_xor_sync(0xffffffffu, warp_min, o));
      // the barrier of the tile before this one (a rescale waits for its P C)
      int before = STAGES - 1, before_parity = 1, stage = 0, parity = 0;
      for (int t = 0; t < n_tiles; ++t) {
        const uint32_t s_addr = tmem + my_lane + COL_S + (t & 1) * TILE_KEYS;
        mbar_wait(&s_done[t & 1], (t >> 1) & 1, status, &gave_up);
        tc_fence_after();
        const int k0 = t * TILE_KEYS;
        float s[TILE_KEYS];
        scores_ld(s_addr, s);
        if (!warp_full || k0 + TILE_KEYS - 1 > warp_min) {
#pragma unroll
          for (int i = 0; i < TILE_KEYS; ++i)
            if (k0 + i > my_pos) s[i] = -INFINITY;
        }
        // four independent chains for the maximum and for the sum
        float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < TILE_KEYS; i += 8) {
          mx4[0] = max3(mx4[0], s[i], s[i + 1]);
          mx4[1] = max3(mx4[1], s[i + 2], s[i + 3]);
          mx4[2] = max3(mx4[2], s[i + 4], s[i + 5]);
          mx4[3] = max3(mx4[3], s[i + 6], s[i + 7]);
        }
        const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
        float alpha = 1.f, sum = 0.f;
        bool raise = false;
        if (mx != -INFINITY && (m_ref == -INFINITY || (mx - m_ref) * c > RESCALE_THRESHOLD)) {
          raise = true;
          alpha = m_ref == -INFINITY ? 0.f : exp2f((m_ref - mx) * c);
          m_ref = mx;
        }
        uint32_t packed[TILE_KEYS / 2];
        if (m_ref == -INFINITY) {
#pragma unroll
          for (int i = 0; i < TILE_KEYS / 2; ++i) packed[i] = 0u;
        } else {
          const float mc = m_ref * c;
          const uint64_t c2 = f32x2(c, c), nmc2 = f32x2(-mc, -mc);
          uint64_t sum2[2] = {f32x2(0.f, 0.f), f32x2(0.f, 0.f)};
#pragma unroll
          for (int i = 0; i < TILE_KEYS; i += 4) {
            float x0, x1, x2, x3;
            f32x2_split(fma_f32x2(f32x2(s[i], s[i + 1]), c2, nmc2), x0, x1);
            f32x2_split(fma_f32x2(f32x2(s[i + 2], s[i + 3]), c2, nmc2), x2, x3);
            const float p0 = ex2_approx(x0), p1 = ex2_approx(x1), p2 = ex2_approx(x2), p3 = ex2_approx(x3);
            sum2[0] = add_f32x2(sum2[0], f32x2(p0, p1));
            sum2[1] = add_f32x2(sum2[1], f32x2(p2, p3));
            packed[i / 2] = pack_bf16(p0, p1);
            packed[i / 2 + 1] = pack_bf16(p2, p3);
          }
          float a0, a1, a2, a3;
          f32x2_split(sum2[0], a0, a1);
          f32x2_split(sum2[1], a2, a3);
          sum = (a0 + a1) + (a2 + a3);
        }
        l_run = l_run * alpha + sum;
        // P_t over the first columns of S_t (this thread has read all of its row)
        probs_st(s_addr, packed);
        // Where a row's reference maximum was raised, O is rescaled before this tile's P C may run, once
        // the P C of the tile before is complete.  (Its barrier completes next for a tile that needs this
        // thread's later probabilities: a wait on it cannot fall behind.)
        if (t > 0 && __any_sync(0xffffffffu, raise)) {
          mbar_wait(&o_done[before], before_parity, status, &gave_up);
          tc_fence_after();
#pragma unroll 1
          for (int cc = 0; cc < RO / 32; ++cc) {
            float part[32];
            tmem_ld32(tmem + my_lane + COL_O + cc * 32, part);
#pragma unroll
            for (int i = 0; i < 32; ++i) part[i] *= alpha;
            tmem_st32(tmem + my_lane + COL_O + cc * 32, part);
          }
        }
        tc_fence_before();
        mbar_arrive(&p_ready[t & 1]);
        before = stage;
        before_parity = parity;
        if (++stage == STAGES) {
          stage = 0;
          parity ^= 1;
        }
      }
      // ---- O / l, times the gate -> out ----
      mbar_wait(&o_done[before], before_parity, status, &gave_up);
      tc_fence_after();
      float f = l_run > 0.f ? 1.f / l_run : 0.f;
      if (gate != nullptr && my_valid)
        f *= 1.f / (1.f + __expf(-__bfloat162float(gate[(size_t)(tok0 + row_token(tid)) * gate_ts + row_head(tid)])));
      __nv_bfloat16* dst = out_row(tid);
#pragma unroll 1
      for (int cc = 0; cc < RO / 32; ++cc) {
        float o[32];
        tmem_ld32(tmem + my_lane + COL_O + cc * 32, o);
        if (my_valid) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            uint4 v;
            v.x = pack_bf16(o[i] * f, o[i + 1] * f);
            v.y = pack_bf16(o[i + 2] * f, o[i + 3] * f);
            v.z = pack_bf16(o[i + 4] * f, o[i + 5] * f);
            v.w = pack_bf16(o[i + 6] * f, o[i + 7] * f);
            *reinterpret_cast<uint4*>(dst + cc * 32 + i) = v;
          }
        }
      }
      tc_fence_before();
    }
  }
  __syncthreads();
  if (*reinterpret_cast<volatile int*>(&gave_up) != 0) {
    // products and copies issued around the wait that ran out may still be running: the block leaves
    // only once they are through (or these waits run out too)
    if (tid == ISSUER * 32) {
      umma_commit(&drained);
      for (int it = 0; it < MBAR_WAIT_POLLS && !mbar_try_wait(&drained, 0); ++it) {
      }
    }
    if (tid == LOADER * 32) {
      const int first = n_tiles > STAGES ? n_tiles - STAGES : 0;
      for (int t = first; t < n_tiles; ++t)
        for (int it = 0; it < MBAR_WAIT_POLLS && !mbar_try_wait(&full[t % STAGES], (t / STAGES) & 1); ++it) {
        }
    }
    __syncthreads();
  }
  if (warp == LOADER) tmem_dealloc(tmem, TMEM);
}

}  // namespace fg_latent_tc5

// map: the layer's pool [pages, 1, page, E] with boxes of min(page, fg_latent_tc5_keys()) rows.  Tiles hold
// 128 / min(heads, 128) tokens each.  Pages of a power of two >= 8 slots.
extern "C" int fg_latent_attention_tc5(const void* map, const void* qa, long qa_ts, long qa_hs, const void* qt, long qt_ts,
                                       long qt_hs, void* out, long out_ts, long out_hs, const void* gate, long gate_ts,
                                       const int* block_table, int table_width, int page_size, int n_pages,
                                       const int* pos, const int* tile_req, const int* tile_tok0, const int* tile_ntok,
                                       int n_tiles, int n_heads, int rank, int rot_dim, int entry, float scale,
                                       int* status, cudaStream_t stream) {
  using namespace fg_latent_tc5;
  if (n_tiles == 0) return 0;
  FG_CHECK_ARG(fg_latent_tc5::SUPPORTED && rank == R && rot_dim == ROT && entry == E,
               "fg_latent_attention_tc5: library built for a latent of %d + %d (entries of %d), got %d + %d (%d)", R, ROT,
               E, rank, rot_dim, entry);
  FG_CHECK_ARG(page_size >= 8 && (page_size & (page_size - 1)) == 0, "fg_latent_attention_tc5: pages of %d slots", page_size);
  FG_CHECK_ARG(((uintptr_t)map & 63) == 0, "fg_latent_attention_tc5: the tensor map must be 64-byte aligned");
  FG_CHECK_ARG(qa_ts % 8 == 0 && qa_hs % 8 == 0 && out_ts % 8 == 0 && out_hs % 8 == 0 && ((uintptr_t)qa & 15) == 0 &&
                   ((uintptr_t)out & 15) == 0,
               "fg_latent_attention_tc5: folded queries and outputs must be 16-byte aligned with strides of 8");
  const int qt_vec = qt_ts % 8 == 0 && qt_hs % 8 == 0 && ((uintptr_t)qt & 15) == 0;
  const int hpb = n_heads < TILE_ROWS ? n_heads : TILE_ROWS;
  const long long blocks = (long long)n_tiles * ((n_heads + hpb - 1) / hpb) * NSPLIT;
  FG_CHECK_ARG(blocks < (1ll << 31), "fg_latent_attention_tc5: %lld blocks", blocks);
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_tc5_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
    FG_CHECK_ARG(e == cudaSuccess, "fg_latent_attention_tc5: shared memory: %s", cudaGetErrorString(e));
    attr_set = true;
  }
  CUtensorMap m;
  memcpy(&m, map, sizeof(m));
  latent_attention_tc5_kernel<<<(unsigned)blocks, N_THREADS, SMEM, stream>>>(
      m, (const __nv_bfloat16*)qa, qa_ts, qa_hs, (const __nv_bfloat16*)qt, qt_ts, qt_hs, qt_vec, (__nv_bfloat16*)out,
      out_ts, out_hs, (const __nv_bfloat16*)gate, gate_ts, block_table, table_width, page_size, n_pages, pos, tile_req,
      tile_tok0, tile_ntok, n_tiles, n_heads, hpb, scale * 1.4426950408889634f, status);
  FG_CHECK_LAUNCH("fg_latent_attention_tc5");
  return 0;
}

#else  // latents of this size have no kernel here

extern "C" int fg_latent_attention_tc5(const void*, const void*, long, long, const void*, long, long, void*, long, long,
                                       const void*, long, const int*, int, int, int, const int*, const int*, const int*,
                                       const int*, int, int, int, int, int, float, int*, cudaStream_t) {
  fg_set_error("fg_latent_attention_tc5: no kernel for a latent of %d numbers", FG_LATENT_RANK);
  return -1;
}

#endif
