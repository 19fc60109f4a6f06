// Attention over a paged latent cache (one latent + one rotated key part per token, shared by all heads).
//
// latent_prepare_kernel   between the projections and the scores: rotation of q and of the shared key part, RMS norm of
//                         the latent, cache store; one CTA per token.
// latent_attn_mma_kernel  bf16, prompts and decode alike.  Queries live in the latent space (the caller multiplied them by
//                         the key up-projection), so every head sees the same keys and a query tile is
//                         (tokens x heads) rows: 16 or 32 rows for a decode step, 64 rows for prompts.  A warp gathers
//                         key tiles from the pages with bulk copies (one key row per lane) into an mbarrier ring; a tile
//                         serves the scores (all kv_rank + rot_dim columns) and the values (its first kv_rank columns).
//                         The other warps form row groups of 16 rows; inside a group they split the reduction of the
//                         scores (each keeps its slice of the queries in registers), then the rows of the softmax, then
//                         the columns of the output, and meet at two named barriers per tile.  Scores, softmax and
//                         accumulators are fp32.  Long key ranges of small batches are split over CTAs and merged by
//                         latent_merge_kernel.
// latent_attn_kernel      any size, any type, one CTA per (token, head); the 32-bit path.
#include "float_common.cuh"
#include "umma.cuh"

namespace b200 {

constexpr int kPage = 16;
constexpr float kLog2e = 1.4426950408889634f;

// ---------------------------------------------------------------------------------------------------
struct PrepareParams {
  const float* qd;
  int splits;
  int64_t split_stride, qd_pitch;
  const int32_t *positions, *out_loc;
  const float* rope;
  int rot_dims, max_pos;
  const float* dkv_norm;
  float eps;
  int heads, dim, rot_dim, kv_rank, head_pitch, qn_pitch, lat_pitch;
  int64_t cache_rows;
};

// Entry i of a rotated vector whose unrotated entries `load` returns.
template <typename F>
__device__ __forceinline__ float rotated(const F& load, int i, int rot_dims, const float* cs) {
  if (i >= rot_dims) return load(i);
  const int half = rot_dims >> 1;
  const int k = i < half ? i : i - half;
  const float c = cs[k], s = cs[half + k];
  return i < half ? load(i) * c - load(i + half) * s : load(i) * c + load(i - half) * s;
}

template <typename T>
__global__ void __launch_bounds__(256)
latent_prepare_kernel(const PrepareParams p, T* __restrict__ qn, T* __restrict__ q_lat, T* __restrict__ cache) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const float* src = p.qd + t * p.qd_pitch;
  auto at = [&](int64_t i) { return part_sum(src + i, p.splits, p.split_stride); };
  const int pos = min(max(p.positions[t], 0), p.max_pos - 1);
  const float* cs = p.rot_dims ? p.rope + (int64_t)pos * p.rot_dims : nullptr;
  const int lat = p.kv_rank + p.rot_dim;
  for (int h = warp; h < p.heads; h += warps) {
    const int64_t q0 = (int64_t)h * p.head_pitch;
    T* n = qn + (t * p.heads + h) * p.qn_pitch;
    for (int i = lane; i < p.dim; i += 32) n[i] = from_f32<T>(at(q0 + i));
    T* r = q_lat + (t * p.heads + h) * p.lat_pitch;
    for (int i = lane; i < p.rot_dim; i += 32)
      r[p.kv_rank + i] = from_f32<T>(rotated([&](int k) { return at(q0 + p.dim + k); }, i, p.rot_dims, cs));
    for (int i = lat + lane; i < p.lat_pitch; i += 32) r[i] = from_f32<T>(0.0f);
  }
  if (!p.dkv_norm) return;
  const int64_t d0 = (int64_t)p.heads * p.head_pitch;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < p.kv_rank; i += blockDim.x) {
    const float v = at(d0 + i);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)p.kv_rank + p.eps);
  const int64_t loc = p.out_loc[t];
  if (loc < 0 || loc >= p.cache_rows) return;
  T* row = cache + loc * p.lat_pitch;
  for (int i = threadIdx.x; i < p.kv_rank; i += blockDim.x) row[i] = from_f32<T>(at(d0 + i) * inv * p.dkv_norm[i]);
  for (int i = threadIdx.x; i < p.rot_dim; i += blockDim.x)
    row[p.kv_rank + i] = from_f32<T>(rotated([&](int k) { return at(d0 + p.kv_rank + k); }, i, p.rot_dims, cs));
}

// ---------------------------------------------------------------------------------------------------
struct AttnParams {
  const int32_t* page_table;
  int64_t table_pitch;
  const int32_t *kv_lens, *seq_start;
  const float* sink;
  int64_t tokens;
  int heads, kv_rank, rot_dim, lat_pitch, out_pitch, window;
  float scale2;                    // scale * log2(e)
  int splits;
  float* ws;                       // splits > 1: [splits][tokens * heads][kv_rank], then [splits][tokens * heads][2]
  int head_groups, heads_per_cta, tokens_per_cta;
};

__device__ __forceinline__ int first_key(int pos, int window) { return window > 0 ? max(pos - window + 1, 0) : 0; }

// Plain form: one CTA of 128 threads per (token, head), 128 keys at a time, online softmax in natural units of log2.
template <typename T>
__global__ void __launch_bounds__(128)
latent_attn_kernel(const AttnParams p, const T* __restrict__ q_lat, const T* __restrict__ cache, T* __restrict__ out, int batch) {
  extern __shared__ float sm[];
  pdl_launch_dependents();
  pdl_wait();
  const int D = p.kv_rank + p.rot_dim;
  float* q = sm;                         // [D]
  float* o = q + D;                      // [kv_rank]
  float* sc = o + p.kv_rank;             // [128]
  float* red = sc + 128;                 // [8]
  const int64_t t = blockIdx.x;
  const int h = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int seq = (int)t, first = (int)t;
  int count = 1;
  if (p.seq_start) {
    int lo = 0, hi = batch;              // the sequence whose range holds token t
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.seq_start[mid] <= t) lo = mid; else hi = mid;
    }
    seq = lo; first = p.seq_start[seq]; count = p.seq_start[seq + 1] - first;
  }
  const int pos = p.kv_lens[seq] - count + (int)(t - first);
  const int32_t* pages = p.page_table + (int64_t)seq * p.table_pitch;
  const T* qs = q_lat + (t * p.heads + h) * p.lat_pitch;
  for (int i = threadIdx.x; i < D; i += 128) q[i] = to_f32(qs[i]);
  for (int i = threadIdx.x; i < p.kv_rank; i += 128) o[i] = 0.0f;
  const float sink2 = p.sink[h] * kLog2e;
  float m = sink2, l = 1.0f;             // the sink is a key without a value whose score is sink2
  __syncthreads();
  for (int k0 = first_key(pos, p.window); k0 <= pos; k0 += 128) {
    const int n = min(128, pos + 1 - k0);
    for (int j = warp; j < n; j += 4) {
      const int key = k0 + j;
      const T* row = cache + ((int64_t)pages[key / kPage] * kPage + key % kPage) * p.lat_pitch;
      float s = 0.0f;
      for (int i = lane; i < D; i += 32) s = fmaf(q[i], to_f32(row[i]), s);
      s = warp_sum(s);
      if (lane == 0) sc[j] = s * p.scale2;
    }
    __syncthreads();
    float v = (int)threadIdx.x < n ? sc[threadIdx.x] : -INFINITY;
    const float wm = warp_maxf(v);
    if (lane == 0) red[warp] = wm;
    __syncthreads();
    const float mn = fmaxf(m, fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])));
    const float alpha = exp2f(m - mn);
    const float e = exp2f(v - mn);
    const float wsum = warp_sum(e);
    if (lane == 0) red[4 + warp] = wsum;
    sc[threadIdx.x] = e;
    __syncthreads();
    l = l * alpha + ((red[4] + red[5]) + (red[6] + red[7]));
    m = mn;
    for (int i = threadIdx.x; i < p.kv_rank; i += 128) {
      float acc = o[i] * alpha;
      for (int j = 0; j < n; ++j) {
        const int key = k0 + j;
        acc = fmaf(sc[j], to_f32(cache[((int64_t)pages[key / kPage] * kPage + key % kPage) * p.lat_pitch + i]), acc);
      }
      o[i] = acc;
    }
    __syncthreads();
  }
  T* dst = out + (t * p.heads + h) * p.out_pitch;
  for (int i = threadIdx.x; i < p.kv_rank; i += 128) dst[i] = from_f32<T>(o[i] / l);
}

// ---------------------------------------------------------------------------------------------------
__device__ __forceinline__ void ldsm_x4(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// MT row groups of 16 query rows, WARPS warps that compute, a ring of STAGES tiles of 32 keys; a warp's
// slice of the reduction has up to KS steps of 16, its slice of the output up to NC pieces of 16 columns.
constexpr int kKeyTile = 32;
constexpr int kScorePitch = kKeyTile + 8;      // values per staged row (fp32 scores, bf16 weights): conflict-free both ways

template <int MT, int WARPS, int STAGES>
struct AttnShape {
  static constexpr int kRows = 16 * MT, kGroup = WARPS / MT;
  static constexpr bool kCopyWarp = WARPS == 4;
  static constexpr int kThreads = 32 * (WARPS + (kCopyWarp ? 1 : 0));
  static size_t smem(int d16) {
    return (size_t)STAGES * kKeyTile * (d16 + 8) * 2 + (size_t)kGroup * kRows * kScorePitch * 4 + (size_t)kRows * kScorePitch * 2 +
           (size_t)3 * kRows * 4 + 2 * STAGES * 8;
  }
};

__device__ __forceinline__ float exp2_approx(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}
__device__ __forceinline__ void bulk_load(unsigned dst, const void* src, unsigned bytes, unsigned bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
__device__ __forceinline__ void group_sync(int group, int threads) {
  asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "r"(threads) : "memory");
}

template <int MT, int WARPS, int STAGES, int KS, int NC, int MINB>
__global__ void __launch_bounds__((AttnShape<MT, WARPS, STAGES>::kThreads), MINB)
latent_attn_mma_kernel(const AttnParams p, const bf16* __restrict__ q_lat, const bf16* __restrict__ cache, bf16* __restrict__ out) {
  using S = AttnShape<MT, WARPS, STAGES>;
  constexpr int R = S::kRows, G = S::kGroup, NK = kKeyTile, RW = 16 / G, U = RW / 4;   // RW: softmax rows per warp
  constexpr bool kCopyWarp = S::kCopyWarp;
  static_assert(G * MT == WARPS && RW % 4 == 0 && (kCopyWarp || STAGES > 2), "shape");
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int D = p.kv_rank + p.rot_dim;
  const int d16 = (D + 15) & ~15, ld = d16 + 8;
  bf16* ks = reinterpret_cast<bf16*>(smem_raw);                              // [STAGES][NK][ld]
  float* sp = reinterpret_cast<float*>(ks + STAGES * NK * ld);               // [G][R][kScorePitch] partial scores
  bf16* ps = reinterpret_cast<bf16*>(sp + G * R * kScorePitch);              // [R][kScorePitch] weights
  float* row_alpha = reinterpret_cast<float*>(ps + R * kScorePitch);         // [R], then [R][2] maximum and sum
  float* row_ml = row_alpha + R;
  uint64_t* bars = reinterpret_cast<uint64_t*>(row_ml + 2 * R);              // full[STAGES], empty[STAGES]

  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const unsigned full0 = smem_u32(bars), empty0 = smem_u32(bars + STAGES);
  const int split = blockIdx.x % p.splits, q_tile = blockIdx.x / p.splits, hg = blockIdx.y, seq = blockIdx.z;
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(full0 + 8 * s, 1);
      mbar_init(empty0 + 8 * s, WARPS);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  for (int r = warp; r < STAGES * NK; r += S::kThreads / 32)                        // columns behind a row's copied part stay zero
    for (int c = p.lat_pitch + lane; c < d16; c += 32) ks[r * ld + c] = __float2bfloat16_rn(0.0f);
  __syncthreads();
  pdl_wait();
  const int start = p.seq_start ? p.seq_start[seq] : seq;
  const int count = p.seq_start ? p.seq_start[seq + 1] - start : 1;
  const int tok0 = q_tile * p.tokens_per_cta;
  if (tok0 >= count) return;
  const int ntok = min(p.tokens_per_cta, count - tok0);
  const int h0 = hg * p.heads_per_cta, nh = min(p.heads_per_cta, p.heads - h0);
  const int rows = ntok * nh;
  const int pos0 = p.kv_lens[seq] - count + tok0;                            // position of the tile's first token
  const int key_lo = first_key(pos0, p.window), key_hi = pos0 + ntok;        // keys [key_lo, key_hi)
  const int all_tiles = (key_hi - key_lo + NK - 1) / NK, per = (all_tiles + p.splits - 1) / p.splits;
  const int tile0 = split * per, tile1 = min(all_tiles, tile0 + per);

  // Copies, one key row per lane and tile; rows behind the last key repeat it (they are masked).  A tile's cache row is
  // looked up one tile ahead.  Small CTAs have a warp for this; the large ones, whose registers an extra warp would cut,
  // let warp 0 do it two tiles before the ring is full again.
  const int32_t* pages = p.page_table + (int64_t)seq * p.table_pitch;
  const unsigned bytes = (unsigned)p.lat_pitch * 2;
  int64_t src_row = 0;
  auto look_up = [&](int tile) {
    if (tile < tile1) {
      const int key = min(key_lo + tile * NK + lane, key_hi - 1);
      src_row = (int64_t)__ldg(pages + key / kPage) * kPage + key % kPage;
    }
  };
  auto copy_tile = [&](int tile) {               // needs look_up(tile); all lanes of one warp; false after an expired wait
    const unsigned i = tile - tile0, s = i % STAGES;
    const int64_t row = src_row;
    look_up(tile + 1);
    if (!__all_sync(FULL_MASK, mbar_wait(empty0 + 8 * s, ((i / STAGES) & 1) ^ 1, 5))) return false;
    if (lane == 0) mbar_expect_tx(full0 + 8 * s, bytes * NK);
    __syncwarp();
    bulk_load(smem_u32(ks + (s * NK + lane) * ld), cache + row * p.lat_pitch, bytes, full0 + 8 * s);
    return true;
  };
  bool ok = true;
  if (kCopyWarp) {
    if (warp == WARPS) {
      look_up(tile0);
      for (int tile = tile0; tile < tile1 && ok; ++tile) ok = copy_tile(tile);
      return;
    }
  } else if (warp == 0) {
    look_up(tile0);
    for (int tile = tile0; tile < min(tile1, tile0 + STAGES - 2) && ok; ++tile) ok = copy_tile(tile);
  }

  const int rg = warp / G, kg = warp % G;
  // this warp's slice of the reduction and its query fragments (row-major A fragments straight from global memory)
  const int k16 = d16 / 16, k_per = (k16 + G - 1) / G, k_lo = kg * k_per, k_n = max(0, min(k_per, k16 - k_lo));
  unsigned qf[KS][4];
  {
    const bf16* src[2];
    bool live[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = rg * 16 + (lane >> 2) + 8 * i, tok = r / nh;
      live[i] = r < rows;
      src[i] = q_lat + ((int64_t)(start + tok0 + (live[i] ? tok : 0)) * p.heads + h0 + (live[i] ? r - tok * nh : 0)) * p.lat_pitch;
    }
#pragma unroll
    for (int i = 0; i < KS; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = (k_lo + i) * 16 + 8 * (j >> 1) + 2 * (lane & 3);
        qf[i][j] = (i < k_n && live[j & 1] && col < p.lat_pitch) ? __ldg(reinterpret_cast<const unsigned*>(src[j & 1] + col)) : 0u;
      }
  }
  // the rows whose softmax this lane works on (eight lanes per row, four keys each), and the keys they may see
  int vis_lo[U], vis_hi[U];
  float m[U], l[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int r = rg * 16 + kg * RW + 4 * u + (lane >> 3), pos = pos0 + r / nh;
    vis_hi[u] = r < rows ? pos : -1;
    vis_lo[u] = p.window > 0 ? pos - p.window + 1 : 0;
    m[u] = -INFINITY;
    l[u] = 0.0f;
  }
  float acc[NC][2][4];
#pragma unroll
  for (int i = 0; i < NC; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[i][j][k] = 0.0f;
  const int c16 = (p.kv_rank + 15) / 16, c_per = (c16 + G - 1) / G;          // 16-column pieces of the output per warp
  const int c_lo = kg * c_per, c_n = max(0, min(c_per, c16 - c_lo));
  const unsigned k_lane = ((lane & 7) + ((lane >> 4) << 3)) * ld + k_lo * 16 + ((lane >> 3) & 1) * 8;
  const unsigned v_lane = (lane & 15) * ld + c_lo * 16 + (lane >> 4) * 8;
  const int frag = (rg * 16 + (lane >> 2)) * kScorePitch + 2 * (lane & 3);
  const unsigned pa = smem_u32(ps + (rg * 16 + (lane & 15)) * kScorePitch + (lane >> 4) * 8);

  for (int tile = tile0; tile < tile1; ++tile) {
    if (!kCopyWarp && warp == 0 && ok && tile + STAGES - 2 < tile1) ok = copy_tile(tile + STAGES - 2);
    const unsigned it = tile - tile0, slot = it % STAGES;
    const bf16* kt = ks + slot * NK * ld;
    if (ok) ok = mbar_wait(full0 + 8 * slot, (it / STAGES) & 1, 6);
    __syncwarp();
    // partial scores: 16 rows x 32 keys over this warp's slice of the reduction
    float s[NK / 8][4];
#pragma unroll
    for (int i = 0; i < NK / 8; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) s[i][k] = 0.0f;
    const unsigned kb = smem_u32(kt + k_lane);
#pragma unroll
    for (int i = 0; i < KS; ++i) {
      if (i < k_n) {
#pragma unroll
        for (int n = 0; n < NK / 16; ++n) {
          unsigned b[4];
          ldsm_x4(b, kb + (unsigned)(n * 16 * ld * 2) + 32 * i);
          mma_bf16(s[2 * n], qf[i], b[0], b[1]);
          mma_bf16(s[2 * n + 1], qf[i], b[2], b[3]);
        }
      }
    }
    float* mine = sp + kg * R * kScorePitch + frag;
#pragma unroll
    for (int i = 0; i < NK / 8; ++i) {
      *reinterpret_cast<float2*>(mine + 8 * i) = make_float2(s[i][0], s[i][1]);
      *reinterpret_cast<float2*>(mine + 8 * kScorePitch + 8 * i) = make_float2(s[i][2], s[i][3]);
    }
    group_sync(rg, 32 * G);
    // softmax step of this warp's rows
    const int key0 = key_lo + tile * NK + 4 * (lane & 7);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int r = rg * 16 + kg * RW + 4 * u + (lane >> 3);
      float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
      for (int g = 0; g < G; ++g) {
        const float4 o = *reinterpret_cast<const float4*>(sp + (g * R + r) * kScorePitch + 4 * (lane & 7));
        v.x += o.x; v.y += o.y; v.z += o.z; v.w += o.w;
      }
      v.x = (key0 <= vis_hi[u] && key0 >= vis_lo[u]) ? v.x * p.scale2 : -INFINITY;
      v.y = (key0 + 1 <= vis_hi[u] && key0 + 1 >= vis_lo[u]) ? v.y * p.scale2 : -INFINITY;
      v.z = (key0 + 2 <= vis_hi[u] && key0 + 2 >= vis_lo[u]) ? v.z * p.scale2 : -INFINITY;
      v.w = (key0 + 3 <= vis_hi[u] && key0 + 3 >= vis_lo[u]) ? v.w * p.scale2 : -INFINITY;
      float mn = fmaxf(fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w)), m[u]);
      mn = fmaxf(mn, __shfl_xor_sync(FULL_MASK, mn, 1));
      mn = fmaxf(mn, __shfl_xor_sync(FULL_MASK, mn, 2));
      mn = fmaxf(mn, __shfl_xor_sync(FULL_MASK, mn, 4));
      const float mu = mn == -INFINITY ? 0.0f : mn;                          // no visible key so far: every weight is 0
      const float alpha = exp2_approx(m[u] - mu);
      m[u] = mn;
      v.x = exp2_approx(v.x - mu); v.y = exp2_approx(v.y - mu); v.z = exp2_approx(v.z - mu); v.w = exp2_approx(v.w - mu);
      l[u] = fmaf(l[u], alpha, (v.x + v.y) + (v.z + v.w));
      *reinterpret_cast<uint2*>(ps + r * kScorePitch + 4 * (lane & 7)) = make_uint2(f32_to_bf16x2(v.x, v.y), f32_to_bf16x2(v.z, v.w));
      if ((lane & 7) == 0) row_alpha[r] = alpha;
    }
    group_sync(rg, 32 * G);
    // output: 16 rows x this warp's columns
    const float a0 = row_alpha[rg * 16 + (lane >> 2)], a1 = row_alpha[rg * 16 + (lane >> 2) + 8];
    if (__any_sync(FULL_MASK, a0 != 1.0f || a1 != 1.0f)) {
#pragma unroll
      for (int i = 0; i < NC; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          acc[i][j][0] *= a0; acc[i][j][1] *= a0;
          acc[i][j][2] *= a1; acc[i][j][3] *= a1;
        }
    }
    const unsigned vb = smem_u32(kt + v_lane);
#pragma unroll
    for (int kk = 0; kk < NK / 16; ++kk) {
      unsigned a[4];
      ldsm_x4(a, pa + 32 * kk);
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        if (i < c_n) {
          unsigned b[4];
          ldsm_x4_t(b, vb + (unsigned)(kk * 16 * ld * 2) + 32 * i);
          mma_bf16(acc[i][0], a, b[0], b[1]);
          mma_bf16(acc[i][1], a, b[2], b[3]);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(empty0 + 8 * slot);
  }
  // maxima and sums to the lanes that hold the output
#pragma unroll
  for (int u = 0; u < U; ++u) {
    l[u] += __shfl_xor_sync(FULL_MASK, l[u], 1);
    l[u] += __shfl_xor_sync(FULL_MASK, l[u], 2);
    l[u] += __shfl_xor_sync(FULL_MASK, l[u], 4);
    if ((lane & 7) == 0) {
      const int r = rg * 16 + kg * RW + 4 * u + (lane >> 3);
      row_ml[2 * r] = m[u];
      row_ml[2 * r + 1] = l[u];
    }
  }
  group_sync(rg, 32 * G);
  if (!ok) {                                      // a copy did not arrive in time (the status word says so): wait for the
    for (int t = max(tile0, tile1 - STAGES); t < tile1; ++t)                 // last ones once more and leave
      mbar_wait(full0 + 8 * ((t - tile0) % STAGES), ((t - tile0) / STAGES) & 1, 6);
    return;
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = rg * 16 + (lane >> 2) + 8 * r;
    if (row >= rows) continue;
    const float mr = row_ml[2 * row], sum = row_ml[2 * row + 1];
    const int tok = row / nh, hd = h0 + row - tok * nh;
    const int64_t gr = (int64_t)(start + tok0 + tok) * p.heads + hd;
    if (p.splits == 1) {
      const float sink2 = __ldg(p.sink + hd) * kLog2e, mf = fmaxf(mr, sink2);
      const float w = exp2f(mr - mf), inv = w / (sum * w + exp2f(sink2 - mf));
      bf16* dst = out + gr * p.out_pitch;
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (i < c_n) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int col = (c_lo + i) * 16 + 8 * j + 2 * (lane & 3);
            const float a = acc[i][j][2 * r] * inv, b = acc[i][j][2 * r + 1] * inv;
            if (col + 1 < p.kv_rank) *reinterpret_cast<unsigned*>(dst + col) = f32_to_bf16x2(a, b);
            else if (col < p.kv_rank) dst[col] = __float2bfloat16_rn(a);
          }
        }
    } else {
      const int64_t all = p.tokens * p.heads;
      float* dst = p.ws + ((int64_t)split * all + gr) * p.kv_rank;
      if (kg == 0 && (lane & 3) == 0) {
        float* ml = p.ws + (int64_t)p.splits * all * p.kv_rank + ((int64_t)split * all + gr) * 2;
        ml[0] = mr;
        ml[1] = sum;
      }
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (i < c_n) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int col = (c_lo + i) * 16 + 8 * j + 2 * (lane & 3);
            if (col < p.kv_rank) dst[col] = acc[i][j][2 * r];
            if (col + 1 < p.kv_rank) dst[col + 1] = acc[i][j][2 * r + 1];
          }
        }
    }
  }
}

// Parts of the key range of one (token, head) row merged, the sink added once.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const AttnParams p, bf16* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t gr = blockIdx.x, all = p.tokens * p.heads;
  const float* ml = p.ws + (int64_t)p.splits * all * p.kv_rank;
  const float sink2 = __ldg(p.sink + gr % p.heads) * kLog2e;
  float m = sink2;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ml[((int64_t)s * all + gr) * 2]);
  float sum = exp2f(sink2 - m);
  for (int s = 0; s < p.splits; ++s) {
    const float* e = ml + ((int64_t)s * all + gr) * 2;
    sum += e[1] * exp2f(e[0] - m);
  }
  const float inv = 1.0f / sum;
  for (int c = threadIdx.x; c < p.kv_rank; c += 128) {
    float v = 0.0f;
    for (int s = 0; s < p.splits; ++s) {
      const float w = exp2f(ml[((int64_t)s * all + gr) * 2] - m);
      if (w > 0.0f) v = fmaf(w, p.ws[((int64_t)s * all + gr) * p.kv_rank + c], v);   // a part without visible keys is skipped
    }
    out[gr * p.out_pitch + c] = __float2bfloat16_rn(v * inv);
  }
}

// ----------------------------------------------------------------------------- host side
// Kernel variants: row groups, consumer warps, ring slots, limits of a warp's slices, CTAs per SM.  A decode step runs on
// small CTAs that share an SM; more than 16 heads with a wide latent become several CTAs whose keys meet in L2.
#define B200_ATTN_VARIANTS(X) \
  X(1, 4, 4, 5, 4, 2) X(1, 4, 2, 9, 8, 2) X(1, 4, 2, 17, 16, 1) \
  X(2, 8, 4, 5, 4, 2) \
  X(4, 8, 4, 5, 4, 1) X(4, 8, 4, 10, 8, 1) X(4, 8, 4, 18, 16, 1)

struct AttnPlan { int mt, warps, stages, ks, nc, minb; };      // mt = 0: the plain kernel

static AttnPlan plan_attn(int max_q, int heads, int kv_rank, int rot_dim) {
  const int d16 = (kv_rank + rot_dim + 15) & ~15, k16 = d16 / 16, c16 = (kv_rank + 15) / 16;
  const int64_t rows = (int64_t)max_q * heads;
  for (int want = rows <= 16 ? 1 : (rows <= 32 ? 2 : 4); want >= 1; want >>= 1) {
#define B200_ATTN_FITS(MT_, W_, ST_, KS_, NC_, MB_)                                                              \
  if (want == MT_ && (k16 + W_ / MT_ - 1) / (W_ / MT_) <= KS_ && (c16 + W_ / MT_ - 1) / (W_ / MT_) <= NC_ &&     \
      AttnShape<MT_, W_, ST_>::smem(d16) <= 227 * 1024)                                                          \
    return {MT_, W_, ST_, KS_, NC_, MB_};
    B200_ATTN_VARIANTS(B200_ATTN_FITS)
#undef B200_ATTN_FITS
  }
  return {0, 0, 0, 0, 0, 0};
}

template <int MT, int WARPS, int STAGES, int KS, int NC, int MINB>
static int launch_mma(const AttnParams& p, const bf16* q, const bf16* cache, bf16* out, dim3 grid, int d16, cudaStream_t st) {
  const size_t smem = AttnShape<MT, WARPS, STAGES>::smem(d16);
  cudaError_t e = cudaFuncSetAttribute(latent_attn_mma_kernel<MT, WARPS, STAGES, KS, NC, MINB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "latent_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  launch_pdl(latent_attn_mma_kernel<MT, WARPS, STAGES, KS, NC, MINB>, grid, dim3(AttnShape<MT, WARPS, STAGES>::kThreads), smem, st, p, q, cache, out);
  return check_launch("latent_attn");
}

static int tiles_for(int max_q, int max_kv, int window, int tokens_per_cta) {
  int64_t span = max_kv;
  if (window > 0 && span > (int64_t)window + tokens_per_cta - 1) span = (int64_t)window + tokens_per_cta - 1;
  return (int)((span + kKeyTile - 1) / kKeyTile);
}

}  // namespace b200

using namespace b200;

extern "C" int b200f_latent_prepare(const float* qd, int splits, int64_t split_stride, int64_t qd_pitch,
                                    const int32_t* positions, const int32_t* out_loc, const float* rope, int rot_dims,
                                    int max_pos, const float* dkv_norm, float eps, void* qn, void* q_lat, void* cache,
                                    int dtype, int64_t tokens, int heads, int dim, int rot_dim, int kv_rank, int head_pitch,
                                    int qn_pitch, int lat_pitch, int64_t cache_rows, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "latent_prepare: dtype %d", dtype);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && heads > 0 && dim >= 0 && rot_dim >= 0 && kv_rank > 0 && splits >= 1 &&
                   head_pitch >= dim + rot_dim && qn_pitch >= dim && lat_pitch >= kv_rank + rot_dim && rot_dims >= 0 &&
                   rot_dims % 2 == 0 && rot_dims <= rot_dim && max_pos > 0 && cache_rows >= 0 &&
                   qd_pitch >= (int64_t)heads * head_pitch + (dkv_norm ? kv_rank + rot_dim : 0),
               B200_E_SHAPE, "latent_prepare: heads=%d dim=%d rot_dim=%d kv_rank=%d rot_dims=%d", heads, dim, rot_dim, kv_rank, rot_dims);
  if (tokens == 0) return B200_OK;
  B200_REQUIRE(qd && positions && qn && q_lat && (!rot_dims || rope) && (!dkv_norm || (cache && out_loc)), B200_E_NULL, "latent_prepare: null pointer");
  PrepareParams p{qd, splits, split_stride, qd_pitch, positions, out_loc, rope, rot_dims, max_pos, dkv_norm, eps, heads, dim, rot_dim,
                  kv_rank, head_pitch, qn_pitch, lat_pitch, cache_rows};
  if (dtype == B200F_BF16)
    launch_pdl(latent_prepare_kernel<bf16>, dim3((unsigned)tokens), dim3(256), 0, (cudaStream_t)s, p, (bf16*)qn, (bf16*)q_lat, (bf16*)cache);
  else
    launch_pdl(latent_prepare_kernel<float>, dim3((unsigned)tokens), dim3(256), 0, (cudaStream_t)s, p, (float*)qn, (float*)q_lat, (float*)cache);
  return check_launch("latent_prepare");
}

extern "C" size_t b200f_latent_attn_ws_floats(int64_t tokens, int heads, int kv_rank, int key_splits) {
  return key_splits > 1 ? (size_t)key_splits * (size_t)tokens * (size_t)heads * ((size_t)kv_rank + 2) : 0;
}

extern "C" int b200f_latent_attn_splits(int64_t tokens, int batch, int max_q, int max_kv, int heads, int kv_rank, int rot_dim,
                                        int window, int dtype) {
  if (dtype != B200F_BF16 || tokens <= 0 || batch <= 0) return 1;
  const AttnPlan pl = plan_attn(max_q, heads, kv_rank, rot_dim);
  if (pl.mt == 0) return 1;
  const int rows = 16 * pl.mt, hpc = heads < rows ? heads : rows, tpc = rows / hpc;
  const int64_t ctas = (int64_t)((max_q + tpc - 1) / tpc) * ((heads + hpc - 1) / hpc) * batch;
  const int tiles = tiles_for(max_q, max_kv, window, tpc);
  int64_t splits = (int64_t)sm_count() * pl.minb / (ctas > 0 ? ctas : 1);
  if (splits > tiles / 4) splits = tiles / 4;                    // a part keeps at least four key tiles
  return (int)(splits < 1 ? 1 : (splits > 32 ? 32 : splits));
}

extern "C" int b200f_latent_attn(const void* q_lat, const void* cache, const int32_t* page_table, int64_t table_pitch,
                                 const int32_t* kv_lens, const int32_t* seq_start, const float* sink, void* out, int dtype,
                                 int64_t tokens, int batch, int max_q, int heads, int kv_rank, int rot_dim, int lat_pitch,
                                 int out_pitch, int window, float scale, int key_splits, float* ws, int simple, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "latent_attn: dtype %d", dtype);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && batch >= 0 && batch < 65536 && max_q > 0 && heads > 0 && heads < 65536 && kv_rank > 0 &&
                   rot_dim >= 0 && lat_pitch >= kv_rank + rot_dim && out_pitch >= kv_rank && window >= 0 && table_pitch > 0 && key_splits >= 1 &&
                   (seq_start || (tokens == batch && max_q == 1)),
               B200_E_SHAPE, "latent_attn: tokens=%lld batch=%d heads=%d kv_rank=%d rot_dim=%d window=%d", (long long)tokens, batch, heads, kv_rank, rot_dim, window);
  if (tokens == 0 || batch == 0) return B200_OK;
  B200_REQUIRE(q_lat && cache && page_table && kv_lens && sink && out && (key_splits == 1 || ws), B200_E_NULL, "latent_attn: null pointer");
  cudaStream_t st = (cudaStream_t)s;
  AttnParams p{page_table, table_pitch, kv_lens, seq_start, sink, tokens, heads, kv_rank, rot_dim, lat_pitch, out_pitch, window,
               scale * kLog2e, key_splits, ws, 1, heads, 1};
  const AttnPlan pl = (dtype == B200F_BF16 && !simple && lat_pitch % 8 == 0 && out_pitch % 2 == 0 && aligned16(q_lat) && aligned16(cache))
                          ? plan_attn(max_q, heads, kv_rank, rot_dim) : AttnPlan{0, 0, 0, 0, 0, 0};
  if (pl.mt == 0) {
    const size_t smem = (size_t)(2 * kv_rank + rot_dim + 128 + 8) * sizeof(float);
    B200_REQUIRE(smem <= 227 * 1024, B200_E_UNSUPPORTED, "latent_attn: kv_rank %d is too large", kv_rank);
    const dim3 grid((unsigned)tokens, (unsigned)heads);
    cudaError_t e = dtype == B200F_BF16
        ? cudaFuncSetAttribute(latent_attn_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
        : cudaFuncSetAttribute(latent_attn_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "latent_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    p.splits = 1;
    if (dtype == B200F_BF16)
      launch_pdl(latent_attn_kernel<bf16>, grid, dim3(128), smem, st, p, (const bf16*)q_lat, (const bf16*)cache, (bf16*)out, batch);
    else
      launch_pdl(latent_attn_kernel<float>, grid, dim3(128), smem, st, p, (const float*)q_lat, (const float*)cache, (float*)out, batch);
    return check_launch("latent_attn (plain)");
  }
  const int rows = 16 * pl.mt, d16 = (kv_rank + rot_dim + 15) & ~15;
  p.heads_per_cta = heads < rows ? heads : rows;
  p.tokens_per_cta = rows / p.heads_per_cta;
  p.head_groups = (heads + p.heads_per_cta - 1) / p.heads_per_cta;
  const int64_t q_tiles = (max_q + p.tokens_per_cta - 1) / p.tokens_per_cta;
  B200_REQUIRE(q_tiles * key_splits < (1ll << 31), B200_E_SHAPE, "latent_attn: too many query tiles");
  const dim3 grid((unsigned)(q_tiles * key_splits), (unsigned)p.head_groups, (unsigned)batch);
  const bf16 *q = (const bf16*)q_lat, *kc = (const bf16*)cache;
  bf16* o = (bf16*)out;
  int rc = B200_E_UNSUPPORTED;
#define B200_ATTN_CASE(MT_, W_, ST_, KS_, NC_, MB_) \
  if (pl.mt == MT_ && pl.ks == KS_ && pl.nc == NC_) rc = launch_mma<MT_, W_, ST_, KS_, NC_, MB_>(p, q, kc, o, grid, d16, st);
  B200_ATTN_VARIANTS(B200_ATTN_CASE)
#undef B200_ATTN_CASE
  if (rc != B200_OK || key_splits == 1) return rc;
  launch_pdl(latent_merge_kernel, dim3((unsigned)(tokens * heads)), dim3(128), 0, st, p, o);
  return check_launch("latent_attn (merge)");
}

extern "C" int b200f_latent_attn_status(int* out_host, int reset) {
  B200_REQUIRE(out_host, B200_E_NULL, "latent_attn_status: null pointer");
  cudaError_t e = cudaMemcpyFromSymbol(out_host, g_gemm_status, sizeof(int));
  if (e == cudaSuccess && reset) {
    const int zero = 0;
    e = cudaMemcpyToSymbol(g_gemm_status, &zero, sizeof(int));
  }
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "latent_attn_status: %s", cudaGetErrorString(e));
  return B200_OK;
}
