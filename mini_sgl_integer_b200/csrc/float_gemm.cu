// Linears of the floating-point models.
//
//   out[b][t, j] = act( sum_k x[b][t, k] * w[b][j, k] )          fp32 accumulation
//
// bf16 operands run on the tensor cores: tcgen05.mma kind::f16 with fp32 accumulators in tensor memory, operands staged
// by TMA into 128-byte-swizzled shared memory (64 values of K per stage row).  Operands are K-major with any row pitch
// that is a multiple of 8 values; K itself is arbitrary (TMA fills the tail with zeros).  A batch index (third TMA
// coordinate) serves the per-head products of latent attention.  Three forms, as for the int8 linears:
//   * decode sizes (M <= 256 tokens): "weights-stationary", 128 weight rows are the UMMA's M side and all tokens its N side,
//     so every weight byte crosses HBM once; with few blocks of weight rows K is split over CTAs, each writing its own
//     fp32 partial matrix (no atomics: the consumer adds the parts in order, so the result is reproducible),
//   * large M: 256 x 256 tiles on CTA pairs (cta_group::2),
//   * in between: one CTA per 128 x BN tile.
// Every wait is bounded as in the int8 kernels.
//
// fp32 operands (B200F_F32) use a plain shared-memory tiled FFMA kernel: true 32-bit products.
#include "float_common.cuh"
#include "umma.cuh"

namespace b200 {

constexpr int kFBM = 128;            // UMMA M side per CTA
constexpr int kFBK = 64;             // bf16 values of K per stage (128 bytes, one swizzle row)
constexpr int kFKBytes = 128;
constexpr int kFEpiWarps = 8;
constexpr int kFThreads = 64 + 32 * kFEpiWarps;
constexpr int kFEpiWarps2 = 16;
constexpr int kFThreads2 = 64 + 32 * kFEpiWarps2;
constexpr int kFStagePitch = 20;     // words per staged row of 16: 16-byte aligned, conflict-free for int4 both ways

struct FGemmParams {
  void* out;
  int out_f32;
  int M, N, K, batch;
  int64_t out_pitch, out_bstride;
  int splits;
  int64_t split_stride;
  int act;
  float act_a, act_b;
  int vec;                           // out rows and batches start on 16-byte boundaries (pitch and strides allow it)
};

__device__ __forceinline__ void umma_bf16(unsigned tmem_d, uint64_t desc_a, uint64_t desc_b, unsigned idesc, unsigned accumulate) {
  asm volatile(
      "{\n.reg .pred p;\n"
      "setp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}"
      ::"r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void umma_bf16_2sm(unsigned tmem_d, uint64_t desc_a, uint64_t desc_b, unsigned idesc, unsigned accumulate) {
  asm volatile(
      "{\n.reg .pred p;\n"
      "setp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::2.kind::f16 [%0], %1, %2, %3, p;\n}"
      ::"r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
// Instruction descriptor of kind::f16: D = f32 (1 << 4), A = B = bf16 (1 << 7, 1 << 10), both K-major, N >> 3 at bit 17,
// M >> 4 at bit 24.
__host__ __device__ constexpr unsigned make_idesc_bf16(int m, int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(n >> 3) << 17) | ((unsigned)(m >> 4) << 24);
}

// One warp's 32 x 32 accumulator chunk (lane = row) to a row-major matrix through a warp-private staging tile, so that
// a store instruction covers whole 64-byte (bf16) or 2 x 64-byte (fp32) row pieces.
__device__ __forceinline__ void f_store_chunk(int* stage, int lane, int (&v)[32], const FGemmParams& p, int64_t boff,
                                              int r_base, int col0) {
  if (p.act == B200F_ACT_XIELU) {
#pragma unroll
    for (int j = 0; j < 32; ++j) v[j] = __float_as_int(xielu_f32(__int_as_float(v[j]), p.act_a, p.act_b));
  }
  if (p.act == B200F_ACT_GATED_SILU) {       // the chunk's first 16 columns are gates, the others what they gate
    bf16* out = reinterpret_cast<bf16*>(p.out) + boff;
    __syncwarp();
#pragma unroll
    for (int j = 0; j < 8; j += 4) {
      unsigned w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int c = 2 * (j + i);
        w[i] = f32_to_bf16x2(silu_f32(__int_as_float(v[c])) * __int_as_float(v[16 + c]), silu_f32(__int_as_float(v[c + 1])) * __int_as_float(v[17 + c]));
      }
      *reinterpret_cast<uint4*>(stage + lane * kFStagePitch + j) = make_uint4(w[0], w[1], w[2], w[3]);
    }
    __syncwarp();
#pragma unroll
    for (int it = 0; it < 2; ++it) {
      const int r = it * 16 + (lane >> 1), row = r_base + r, col = (col0 >> 1) + 8 * (lane & 1), n = p.N >> 1;
      if (row < p.M && col < n) {
        const uint4 o = *reinterpret_cast<const uint4*>(stage + r * kFStagePitch + 4 * (lane & 1));
        bf16* dst = out + (int64_t)row * p.out_pitch + col;
        if (p.vec && col + 7 < n) {
          *reinterpret_cast<uint4*>(dst) = o;
        } else {
          const unsigned w[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
          for (int i = 0; i < 8; ++i)
            if (col + i < n) reinterpret_cast<unsigned short*>(dst)[i] = (unsigned short)(w[i >> 1] >> (16 * (i & 1)));
        }
      }
    }
    return;
  }
  const int rr = lane >> 2, cc = (lane & 3) * 4;
  if (p.out_f32) {
    float* out = reinterpret_cast<float*>(p.out) + boff;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      __syncwarp();
#pragma unroll
      for (int j = 0; j < 16; j += 4)
        *reinterpret_cast<int4*>(stage + lane * kFStagePitch + j) = make_int4(v[16 * h + j], v[16 * h + j + 1], v[16 * h + j + 2], v[16 * h + j + 3]);
      __syncwarp();
#pragma unroll
      for (int it = 0; it < 4; ++it) {
        const int r = it * 8 + rr, row = r_base + r, col = col0 + 16 * h + cc;
        if (row < p.M && col < p.N) {
          const int4 o = *reinterpret_cast<const int4*>(stage + r * kFStagePitch + cc);
          int* dst = reinterpret_cast<int*>(out + (int64_t)row * p.out_pitch + col);
          if (p.vec && col + 3 < p.N) {
            *reinterpret_cast<int4*>(dst) = o;
          } else {
            dst[0] = o.x;
            if (col + 1 < p.N) dst[1] = o.y;
            if (col + 2 < p.N) dst[2] = o.z;
            if (col + 3 < p.N) dst[3] = o.w;
          }
        }
      }
    }
  } else {
    bf16* out = reinterpret_cast<bf16*>(p.out) + boff;
    __syncwarp();
#pragma unroll
    for (int j = 0; j < 16; j += 4) {
      unsigned w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) w[i] = f32_to_bf16x2(__int_as_float(v[2 * (j + i)]), __int_as_float(v[2 * (j + i) + 1]));
      *reinterpret_cast<uint4*>(stage + lane * kFStagePitch + j) = make_uint4(w[0], w[1], w[2], w[3]);
    }
    __syncwarp();
#pragma unroll
    for (int it = 0; it < 4; ++it) {
      const int r = it * 8 + rr, row = r_base + r, col = col0 + 2 * cc;
      if (row < p.M && col < p.N) {
        const uint4 o = *reinterpret_cast<const uint4*>(stage + r * kFStagePitch + cc);
        bf16* dst = out + (int64_t)row * p.out_pitch + col;
        if (p.vec && col + 7 < p.N) {
          *reinterpret_cast<uint4*>(dst) = o;
        } else {
          const unsigned w[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
          for (int i = 0; i < 8; ++i)
            if (col + i < p.N) reinterpret_cast<unsigned short*>(dst)[i] = (unsigned short)(w[i >> 1] >> (16 * (i & 1)));
        }
      }
    }
  }
}

// Weights-stationary tiles: batch-major, then blocks of 128 weight rows, then parts of K.
struct FWsTile { int b, n_blk, part, kb0, kb1; };
__device__ __forceinline__ FWsTile f_ws_tile(const FGemmParams& p, int tile, int n_blocks, int num_kb) {
  FWsTile t;
  t.part = tile % p.splits;
  const int r = tile / p.splits;
  t.n_blk = r % n_blocks;
  t.b = r / n_blocks;
  const int per = (num_kb + p.splits - 1) / p.splits;
  t.kb0 = t.part * per;
  t.kb1 = min(num_kb, t.kb0 + per);
  return t;
}

template <int BN, int STAGES, bool WS>
__global__ void __launch_bounds__(kFThreads, 1)
gemm_bf16_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b, const FGemmParams p) {
  extern __shared__ __align__(1024) unsigned char smem[];
  constexpr int kABytes = kFBM * kFKBytes;
  constexpr int kBBytes = BN * kFKBytes;
  constexpr int kStageBytes = kABytes + kBBytes;
  unsigned char* tiles = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(tiles + STAGES * kStageBytes);   // full[S], empty[S], tfull[2], tempty[2]
  unsigned* tmem_slot = reinterpret_cast<unsigned*>(bars + 2 * STAGES + 4);
  int* stage_all = reinterpret_cast<int*>(tmem_slot + 4);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int num_kb = (p.K + kFBK - 1) / kFBK;
  const int m_tiles = WS ? 1 : (p.M + kFBM - 1) / kFBM;
  const int n_tiles = WS ? (p.N + kFBM - 1) / kFBM : (p.N + BN - 1) / BN;
  const int num_tiles = p.batch * n_tiles * (WS ? p.splits : m_tiles);
  const unsigned full0 = smem_u32(bars), empty0 = smem_u32(bars + STAGES);
  const unsigned tfull0 = smem_u32(bars + 2 * STAGES), tempty0 = smem_u32(bars + 2 * STAGES + 2);

  if (warp == 0 && lane == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(full0 + 8 * s, 1);
      mbar_init(empty0 + 8 * s, 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(tfull0 + 8 * s, 1);
      mbar_init(tempty0 + 8 * s, kFEpiWarps);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(2 * BN) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_launch_dependents();
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const unsigned tmem_base = *tmem_slot;
  pdl_wait();

  // tile -> (batch, weight block, token block or part of K)
  auto decode_tile = [&](int tile) {
    if (WS) return f_ws_tile(p, tile, n_tiles, num_kb);
    FWsTile t;
    t.part = tile % m_tiles;                        // token block
    const int r = tile / m_tiles;
    t.n_blk = r % n_tiles;
    t.b = r / n_tiles;
    t.kb0 = 0; t.kb1 = num_kb;
    return t;
  };

  if (warp == 0) {
    if (lane == 0) {
      unsigned it = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        const FWsTile t = decode_tile(tile);
        for (int kb = t.kb0; kb < t.kb1; ++kb, ++it) {
          const unsigned s = it % STAGES, ph = (it / STAGES) & 1;
          ok = mbar_wait(empty0 + 8 * s, ph ^ 1, 1);
          if (!ok) break;
          mbar_expect_tx(full0 + 8 * s, kStageBytes);
          const unsigned a_dst = smem_u32(tiles + s * kStageBytes);
          // map_a feeds the 128-row operand: token rows, or weight rows in the weights-stationary form
          tma_load_3d(a_dst, &map_a, kb * kFBK, (WS ? t.n_blk : t.part) * kFBM, t.b, full0 + 8 * s);
          tma_load_3d(a_dst + kABytes, &map_b, kb * kFBK, WS ? 0 : t.n_blk * BN, t.b, full0 + 8 * s);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr unsigned idesc = make_idesc_bf16(kFBM, BN);
      unsigned it = 0, lt = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x, ++lt) {
        const unsigned slot = lt & 1, aph = (lt >> 1) & 1;
        ok = mbar_wait(tempty0 + 8 * slot, aph ^ 1, 4);
        if (!ok) break;
        tcgen05_fence_after();
        const unsigned tmem_d = tmem_base + slot * BN;
        const FWsTile t = decode_tile(tile);
        for (int kb = t.kb0; kb < t.kb1; ++kb, ++it) {
          const unsigned s = it % STAGES, ph = (it / STAGES) & 1;
          ok = mbar_wait(full0 + 8 * s, ph, 2);
          if (!ok) break;
          tcgen05_fence_after();
          const unsigned a_addr = smem_u32(tiles + s * kStageBytes);
          const uint64_t da = make_smem_desc(a_addr), db = make_smem_desc(a_addr + kABytes);
#pragma unroll
          for (int k = 0; k < 4; ++k)      // 16 values = 32 bytes of K per MMA
            umma_bf16(tmem_d, da + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc, (kb > t.kb0 || k > 0) ? 1u : 0u);
          tcgen05_commit(empty0 + 8 * s);
        }
        if (ok) tcgen05_commit(tfull0 + 8 * slot);
      }
    }
  } else {
    const int q = warp & 3;
    const int half = (warp - 2) >> 2;
    int* stage = stage_all + (warp - 2) * (32 * kFStagePitch);
    unsigned lt = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < num_tiles; tile += gridDim.x, ++lt) {
      const FWsTile t = decode_tile(tile);
      const unsigned slot = lt & 1, aph = (lt >> 1) & 1;
      if (ok) ok = mbar_wait(tfull0 + 8 * slot, aph, 3);
      __syncwarp();
      tcgen05_fence_after();
      if (WS) {
        const int ch = t.n_blk * kFBM + q * 32 + lane;         // rows of the accumulator are weight rows, columns tokens
        const int64_t off = (int64_t)t.b * p.out_bstride + (int64_t)t.part * p.split_stride + ch;
#pragma unroll 1
        for (int c0 = half * 32; c0 < BN; c0 += 64) {
          if (c0 >= p.M) break;
          int v[32];
          tmem_ld_32x32(tmem_base + ((unsigned)(q * 32) << 16) + slot * BN + (unsigned)c0, v);
          if (p.act == B200F_ACT_GATED_SILU) {                   // weight rows alternate: 16 gates, 16 gated
            bf16* out = reinterpret_cast<bf16*>(p.out) + (int64_t)t.b * p.out_bstride + ((ch >> 5) * 16 + (ch & 15));
#pragma unroll
            for (int j = 0; j < 32; ++j) {
              const float up = __int_as_float(__shfl_down_sync(FULL_MASK, v[j], 16));
              if (ok && lane < 16 && ch < p.N && c0 + j < p.M)
                out[(int64_t)(c0 + j) * p.out_pitch] = __float2bfloat16_rn(silu_f32(__int_as_float(v[j])) * up);
            }
          } else if (ok && ch < p.N) {
            if (p.act == B200F_ACT_XIELU) {
#pragma unroll
              for (int j = 0; j < 32; ++j) v[j] = __float_as_int(xielu_f32(__int_as_float(v[j]), p.act_a, p.act_b));
            }
            if (p.out_f32) {
              float* out = reinterpret_cast<float*>(p.out) + off;
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (c0 + j < p.M) out[(int64_t)(c0 + j) * p.out_pitch] = __int_as_float(v[j]);
            } else {
              bf16* out = reinterpret_cast<bf16*>(p.out) + off;
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (c0 + j < p.M) out[(int64_t)(c0 + j) * p.out_pitch] = __float2bfloat16_rn(__int_as_float(v[j]));
            }
          }
          __syncwarp();
        }
      } else {
        const int r_base = t.part * kFBM + q * 32;
#pragma unroll 1
        for (int c0 = half * 32; c0 < BN; c0 += 64) {
          const int col0 = t.n_blk * BN + c0;
          if (col0 >= p.N) break;
          int v[32];
          tmem_ld_32x32(tmem_base + ((unsigned)(q * 32) << 16) + slot * BN + (unsigned)c0, v);
          if (ok) f_store_chunk(stage, lane, v, p, (int64_t)t.b * p.out_bstride, r_base, col0);
        }
      }
      tcgen05_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(tempty0 + 8 * slot);
    }
  }
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(2 * BN) : "memory");
  }
}

// 256 x 256 tiles on CTA pairs; the protocol of the two-CTA int8 kernel.
template <int STAGES>
__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(kFThreads2, 1)
gemm_bf16_2sm_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b, const FGemmParams p) {
  constexpr int BN = 256;
  constexpr int kABytes = kFBM * kFKBytes;
  constexpr int kBBytes = (BN / 2) * kFKBytes;
  constexpr int kStageBytes = kABytes + kBBytes;
  extern __shared__ __align__(1024) unsigned char smem[];
  unsigned char* tiles = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(tiles + STAGES * kStageBytes);
  unsigned* tmem_slot = reinterpret_cast<unsigned*>(bars + 2 * STAGES + 4);
  int* stage_all = reinterpret_cast<int*>(tmem_slot + 4);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  unsigned rank;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(rank));
  const bool leader = rank == 0;
  const int pair = blockIdx.x >> 1, num_pairs = gridDim.x >> 1;
  const int num_kb = (p.K + kFBK - 1) / kFBK;
  const int m_tiles = (p.M + 2 * kFBM - 1) / (2 * kFBM), n_tiles = (p.N + BN - 1) / BN;
  const int num_tiles = p.batch * m_tiles * n_tiles;
  const unsigned full0 = smem_u32(bars), empty0 = smem_u32(bars + STAGES);
  const unsigned tfull0 = smem_u32(bars + 2 * STAGES), tempty0 = smem_u32(bars + 2 * STAGES + 2);

  if (warp == 0 && lane == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(full0 + 8 * s, 1);
      mbar_init(empty0 + 8 * s, 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(tfull0 + 8 * s, 1);
      mbar_init(tempty0 + 8 * s, 2 * kFEpiWarps2);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(2 * BN) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;" ::: "memory");
  }
  pdl_launch_dependents();
  tcgen05_fence_before();
  __syncthreads();
  cluster_barrier();
  tcgen05_fence_after();
  const unsigned tmem_base = *tmem_slot;
  pdl_wait();

  if (warp == 0) {
    if (lane == 0) {
      unsigned it = 0;
      bool ok = true;
      for (int tile = pair; tile < num_tiles && ok; tile += num_pairs) {
        const int m_blk = tile % m_tiles, r = tile / m_tiles, n_blk = r % n_tiles, b = r / n_tiles;
        for (int kb = 0; kb < num_kb; ++kb, ++it) {
          const unsigned s = it % STAGES, ph = (it / STAGES) & 1;
          ok = mbar_wait(empty0 + 8 * s, ph ^ 1, 1);
          if (!ok) break;
          if (leader) mbar_expect_tx(full0 + 8 * s, 2 * kStageBytes);
          const unsigned a_dst = smem_u32(tiles + s * kStageBytes);
          const unsigned lbar = (full0 + 8 * s) & kPeerBitMask;
          tma_load_3d_2sm(a_dst, &map_a, kb * kFBK, m_blk * 2 * kFBM + (int)rank * kFBM, b, lbar);
          tma_load_3d_2sm(a_dst + kABytes, &map_b, kb * kFBK, n_blk * BN + (int)rank * (BN / 2), b, lbar);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && leader) {
      constexpr unsigned idesc = make_idesc_bf16(2 * kFBM, BN);
      unsigned it = 0, lt = 0;
      bool ok = true;
      for (int tile = pair; tile < num_tiles && ok; tile += num_pairs, ++lt) {
        const unsigned slot = lt & 1, aph = (lt >> 1) & 1;
        ok = mbar_wait(tempty0 + 8 * slot, aph ^ 1, 4);
        if (!ok) break;
        tcgen05_fence_after();
        const unsigned tmem_d = tmem_base + slot * BN;
        for (int kb = 0; kb < num_kb; ++kb, ++it) {
          const unsigned s = it % STAGES, ph = (it / STAGES) & 1;
          ok = mbar_wait(full0 + 8 * s, ph, 2);
          if (!ok) break;
          tcgen05_fence_after();
          const unsigned a_addr = smem_u32(tiles + s * kStageBytes);
          const uint64_t da = make_smem_desc(a_addr), db = make_smem_desc(a_addr + kABytes);
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_2sm(tmem_d, da + (uint64_t)(2 * k), db + (uint64_t)(2 * k), idesc, (kb > 0 || k > 0) ? 1u : 0u);
          tcgen05_commit_pair(empty0 + 8 * s);
        }
        if (ok) tcgen05_commit_pair(tfull0 + 8 * slot);
      }
    }
  } else {
    const int q = warp & 3;
    const int part = (warp - 2) >> 2;
    int* stage = stage_all + (warp - 2) * (32 * kFStagePitch);
    unsigned lt = 0;
    bool ok = true;
    for (int tile = pair; tile < num_tiles; tile += num_pairs, ++lt) {
      const int m_blk = tile % m_tiles, r = tile / m_tiles, n_blk = r % n_tiles, b = r / n_tiles;
      const unsigned slot = lt & 1, aph = (lt >> 1) & 1;
      const int r_base = m_blk * 2 * kFBM + (int)rank * kFBM + q * 32;
      if (ok) ok = mbar_wait(tfull0 + 8 * slot, aph, 3);
      __syncwarp();
      tcgen05_fence_after();
#pragma unroll 1
      for (int c0 = part * 32; c0 < BN; c0 += 32 * (kFEpiWarps2 / 4)) {
        const int col0 = n_blk * BN + c0;
        if (col0 >= p.N) break;
        int v[32];
        tmem_ld_32x32(tmem_base + ((unsigned)(q * 32) << 16) + slot * BN + (unsigned)c0, v);
        if (ok) f_store_chunk(stage, lane, v, p, (int64_t)b * p.out_bstride, r_base, col0);
      }
      tcgen05_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive_leader(tempty0 + 8 * slot);
    }
  }
  tcgen05_fence_before();
  __syncthreads();
  cluster_barrier();
  if (warp == 1) {
    tcgen05_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(2 * BN) : "memory");
  }
}

// ----------------------------------------------------------------------------- true 32-bit linears
// 64 x 64 outputs per CTA, 4 x 4 per thread, K in steps of 16 through shared memory.
__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, const FGemmParams p, int64_t x_pitch,
                int64_t x_bstride, int64_t w_pitch, int64_t w_bstride) {
  __shared__ float xs[16][68], ws[16][68];
  pdl_launch_dependents();
  pdl_wait();
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, b = blockIdx.z;
  x += (int64_t)b * x_bstride;
  w += (int64_t)b * w_bstride;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
    const int kk = threadIdx.x & 15, r0 = threadIdx.x >> 4;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + 16 * i;
      xs[kk][r] = (m0 + r < p.M && k0 + kk < p.K) ? x[(int64_t)(m0 + r) * x_pitch + k0 + kk] : 0.0f;
      ws[kk][r] = (n0 + r < p.N && k0 + kk < p.K) ? w[(int64_t)(n0 + r) * w_pitch + k0 + kk] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 c = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, cv[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], cv[j], acc[i][j]);
    }
    __syncthreads();
  }
  float* out = reinterpret_cast<float*>(p.out) + (int64_t)b * p.out_bstride;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < p.M && n < p.N)
        out[(int64_t)m * p.out_pitch + n] = p.act == B200F_ACT_XIELU ? xielu_f32(acc[i][j], p.act_a, p.act_b) : acc[i][j];
    }
}

// ----------------------------------------------------------------------------- host side
// bf16 operand [batch][rows, K] (pitches in values, multiples of 8); box = 64 values of K x box_rows rows, 128-byte swizzle.
static bool make_map_bf16(CUtensorMap* map, const void* base, int64_t rows, int64_t K, int64_t batch, int64_t pitch,
                          int64_t bstride, int box_rows) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return false;
  const cuuint64_t dims[3] = {(cuuint64_t)K, (cuuint64_t)rows, (cuuint64_t)batch};
  const cuuint64_t strides[2] = {(cuuint64_t)pitch * 2, (cuuint64_t)(batch > 1 ? bstride : pitch) * 2};
  const cuuint32_t box[3] = {(cuuint32_t)kFBK, (cuuint32_t)box_rows, 1};
  const cuuint32_t estr[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BN, int STAGES, bool WS>
static int launch_bf16(const CUtensorMap& ma, const CUtensorMap& mb, const FGemmParams& p, cudaStream_t st) {
  constexpr size_t smem = (size_t)STAGES * (kFBM + BN) * kFKBytes + 1024 + (2 * STAGES + 4) * 8 + 16 + kFEpiWarps * 32 * kFStagePitch * 4;
  static_assert(smem <= 227 * 1024, "shared memory budget");
  cudaError_t e = cudaFuncSetAttribute(gemm_bf16_kernel<BN, STAGES, WS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "gemm: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  const int64_t tiles = (int64_t)p.batch * (WS ? (int64_t)((p.N + kFBM - 1) / kFBM) * p.splits
                                               : (int64_t)((p.N + BN - 1) / BN) * ((p.M + kFBM - 1) / kFBM));
  const int grid = (int)(tiles < sm_count() ? tiles : sm_count());
  launch_pdl(gemm_bf16_kernel<BN, STAGES, WS>, dim3(grid), dim3(kFThreads), smem, st, ma, mb, p);
  return check_launch("gemm (bf16)");
}

template <int STAGES>
static int launch_bf16_2sm(const CUtensorMap& ma, const CUtensorMap& mb, const FGemmParams& p, cudaStream_t st) {
  constexpr size_t smem = (size_t)STAGES * 256 * kFKBytes + 1024 + (2 * STAGES + 4) * 8 + 16 + kFEpiWarps2 * 32 * kFStagePitch * 4;
  static_assert(smem <= 227 * 1024, "shared memory budget");
  cudaError_t e = cudaFuncSetAttribute(gemm_bf16_2sm_kernel<STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "gemm: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  const int64_t tiles = (int64_t)p.batch * ((p.N + 255) / 256) * ((p.M + 255) / 256);
  const int pairs = (int)(tiles < sm_count() / 2 ? tiles : sm_count() / 2);
  launch_pdl(gemm_bf16_2sm_kernel<STAGES>, dim3(2 * pairs), dim3(kFThreads2), smem, st, ma, mb, p);
  return check_launch("gemm (bf16, two-CTA tiles)");
}

static bool is_decode_size(int64_t m) { return m <= 256; }

}  // namespace b200

using namespace b200;

extern "C" int b200f_gemm_splits(int64_t m, int64_t n, int64_t k, int64_t batch, int dtype) {
  if (dtype != B200F_BF16 || !is_decode_size(m) || m <= 0 || n <= 0 || k <= 0 || batch <= 0) return 1;
  const int64_t blocks = batch * ((n + kFBM - 1) / kFBM), num_kb = (k + kFBK - 1) / kFBK;
  int splits = (int)(blocks < sm_count() ? sm_count() / blocks : 1);
  splits = splits < 1 ? 1 : (splits > 6 ? 6 : splits);      // beyond six the consumer's reading of the parts costs more
  while (splits > 1 && num_kb / splits < 4) --splits;
  while (splits > 1 && (splits - 1) * ((num_kb + splits - 1) / splits) >= num_kb) --splits;   // no empty part
  return splits;
}

extern "C" int b200f_gemm(const void* x, const void* w, void* out, int dtype, int out_f32, int64_t m, int64_t n, int64_t k,
                          int64_t batch, int64_t x_pitch, int64_t x_bstride, int64_t w_pitch, int64_t w_bstride,
                          int64_t out_pitch, int64_t out_bstride, int splits, int64_t split_stride, int act, float act_a,
                          float act_b, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "gemm: dtype %d", dtype);
  B200_REQUIRE(x && w && out, B200_E_NULL, "gemm: null pointer");
  B200_REQUIRE(m >= 0 && n > 0 && k > 0 && batch > 0 && m < (1ll << 31) && n < (1ll << 31) && k < (1ll << 31) && batch < (1 << 16),
               B200_E_SHAPE, "gemm: m=%lld n=%lld k=%lld batch=%lld", (long long)m, (long long)n, (long long)k, (long long)batch);
  B200_REQUIRE(x_pitch >= k && w_pitch >= k && out_pitch >= (act == B200F_ACT_GATED_SILU ? n / 2 : n), B200_E_SHAPE, "gemm: a row pitch is shorter than its row");
  B200_REQUIRE(act == B200F_ACT_NONE || act == B200F_ACT_XIELU || (act == B200F_ACT_GATED_SILU && dtype == B200F_BF16 && !out_f32 && n % 32 == 0),
               B200_E_UNSUPPORTED, "gemm: activation %d", act);
  B200_REQUIRE(splits >= 1 && (splits == 1 || (act == B200F_ACT_NONE && out_f32 && dtype == B200F_BF16 && is_decode_size(m))),
               B200_E_UNSUPPORTED, "gemm: splits=%d needs a 32-bit output without activation at decode sizes", splits);
  if (m == 0) return B200_OK;
  cudaStream_t st = (cudaStream_t)s;
  FGemmParams p;
  p.out = out; p.out_f32 = out_f32 || dtype == B200F_F32; p.M = (int)m; p.N = (int)n; p.K = (int)k; p.batch = (int)batch;
  p.out_pitch = out_pitch; p.out_bstride = out_bstride; p.splits = splits; p.split_stride = split_stride;
  p.act = act; p.act_a = act_a; p.act_b = act_b;
  if (dtype == B200F_F32) {
    const dim3 grid((unsigned)((n + 63) / 64), (unsigned)((m + 63) / 64), (unsigned)batch);
    B200_REQUIRE(grid.y < 65536 && grid.z < 65536, B200_E_SHAPE, "gemm: too many rows or batches");
    launch_pdl(gemm_f32_kernel, grid, dim3(256), 0, st, (const float*)x, (const float*)w, p, x_pitch, x_bstride, w_pitch, w_bstride);
    return check_launch("gemm (fp32)");
  }
  B200_REQUIRE(aligned16(x) && aligned16(w), B200_E_ALIGN, "gemm: operands must be 16-byte aligned");
  B200_REQUIRE(x_pitch % 8 == 0 && w_pitch % 8 == 0 && (batch == 1 || (x_bstride % 8 == 0 && w_bstride % 8 == 0)), B200_E_ALIGN,
               "gemm: operand pitches and batch strides must be multiples of 8 values");
  const int ev = p.out_f32 ? 4 : 8;
  p.vec = aligned16(out) && out_pitch % ev == 0 && (batch == 1 || out_bstride % ev == 0);
  const int num_kb = (int)((k + kFBK - 1) / kFBK);
  B200_REQUIRE(splits <= num_kb && (splits - 1) * ((num_kb + splits - 1) / splits) < num_kb, B200_E_SHAPE,
               "gemm: %d parts of K leave one empty", splits);
  CUtensorMap ma, mb;
  const bool few_blocks = batch * ((n + kFBM - 1) / kFBM) < 2 * sm_count();
  if (m <= 128 || (is_decode_size(m) && (few_blocks || splits > 1))) {
    const int bn = m <= 32 ? 32 : (m <= 64 ? 64 : (m <= 128 ? 128 : 256));
    B200_REQUIRE(make_map_bf16(&ma, w, n, k, batch, w_pitch, w_bstride, kFBM) && make_map_bf16(&mb, x, m, k, batch, x_pitch, x_bstride, bn),
                 B200_E_CUDA, "gemm: cuTensorMapEncodeTiled failed");
    switch (bn) {
      case 256: return launch_bf16<256, 4, true>(ma, mb, p, st);
      case 128: return launch_bf16<128, 6, true>(ma, mb, p, st);
      case 64: return launch_bf16<64, 8, true>(ma, mb, p, st);
      default: return launch_bf16<32, 9, true>(ma, mb, p, st);
    }
  }
  B200_REQUIRE(make_map_bf16(&ma, x, m, k, batch, x_pitch, x_bstride, kFBM), B200_E_CUDA, "gemm: cuTensorMapEncodeTiled failed");
  if (batch * ((m + 255) / 256) * ((n + 255) / 256) >= sm_count() / 2) {
    B200_REQUIRE(make_map_bf16(&mb, w, n, k, batch, w_pitch, w_bstride, kFBM), B200_E_CUDA, "gemm: cuTensorMapEncodeTiled failed");
    return launch_bf16_2sm<5>(ma, mb, p, st);
  }
  const int64_t m_tiles = (m + kFBM - 1) / kFBM;
  int bn = 256;
  while (bn > 32 && batch * m_tiles * ((n + bn - 1) / bn) < sm_count()) bn >>= 1;
  B200_REQUIRE(make_map_bf16(&mb, w, n, k, batch, w_pitch, w_bstride, bn), B200_E_CUDA, "gemm: cuTensorMapEncodeTiled failed");
  switch (bn) {
    case 256: return launch_bf16<256, 4, false>(ma, mb, p, st);
    case 128: return launch_bf16<128, 6, false>(ma, mb, p, st);
    case 64: return launch_bf16<64, 8, false>(ma, mb, p, st);
    default: return launch_bf16<32, 9, false>(ma, mb, p, st);
  }
}

extern "C" int b200f_gemm_status(int* out_host, int reset) {
  B200_REQUIRE(out_host, B200_E_NULL, "gemm_status: null pointer");
  cudaError_t e = cudaMemcpyFromSymbol(out_host, g_gemm_status, sizeof(int));
  if (e == cudaSuccess && reset) {
    const int zero = 0;
    e = cudaMemcpyToSymbol(g_gemm_status, &zero, sizeof(int));
  }
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "gemm_status: %s", cudaGetErrorString(e));
  return B200_OK;
}
