// Attention over a paged latent cache (one latent + one rotated key part per token, shared by all heads).
//
// latent_prepare_kernel   between the projections and the scores: rotation of q and of the shared key part, RMS norm of
//                         the latent, cache store; one CTA per token.
// latent_attn_mma_kernel  bf16, prompts and decode alike.  Queries live in the latent space (the caller multiplied them by
//                         the key up-projection), so every head sees the same keys and a query tile is
//                         (tokens x heads) rows: 16 rows for a decode step with few heads, 64 rows for prompts.  Key tiles
//                         are gathered from the pages with cp.async into a double buffer; a tile serves the scores (all
//                         kv_rank + rot_dim columns) and the values (its first kv_rank columns).  Eight warps: the scores are
//                         split over (row groups x key groups), the output over (row groups x column groups), with the
//                         probabilities exchanged through shared memory.  Scores, softmax and accumulators are fp32.
//                         Long key ranges of small batches are split over CTAs and merged by latent_merge_kernel.
// latent_attn_kernel      any size, any type, one CTA per (token, head); the 32-bit path.
#include "float_common.cuh"

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
__device__ __forceinline__ unsigned sm_addr(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(unsigned dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm_x4(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x2(unsigned& r0, unsigned& r1, unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// MT row groups of 16 query rows, NK keys per tile, up to NC16 16-column pieces of the output per warp.
template <int MT, int NK>
struct AttnShape {
  static constexpr int kRows = 16 * MT, kGroups = 8 / MT, kKeysPerWarp = NK / kGroups;
  static constexpr int kPPitch = NK + 8;                                     // bf16, conflict-free for ldmatrix
  static size_t smem(int d16) {
    return (size_t)(kRows + 2 * NK) * (d16 + 8) * 2 + (size_t)kRows * kPPitch * 2 + (size_t)2 * kRows * kGroups * 4;
  }
};

template <int MT, int NK, int NC16>
__global__ void __launch_bounds__(256)
latent_attn_mma_kernel(const AttnParams p, const bf16* __restrict__ q_lat, const bf16* __restrict__ cache, bf16* __restrict__ out) {
  using S = AttnShape<MT, NK>;
  constexpr int R = S::kRows, G = S::kGroups, KW = S::kKeysPerWarp, KT = KW / 8;
  static_assert(KW >= 8 && KW % 8 == 0, "key tile too small for this many warps");
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int D = p.kv_rank + p.rot_dim;
  const int d16 = (D + 15) & ~15, ld = d16 + 8;
  bf16* qs = reinterpret_cast<bf16*>(smem_raw);                              // [R][ld]
  bf16* ks = qs + R * ld;                                                    // [2][NK][ld]
  bf16* ps = ks + 2 * NK * ld;                                               // [R][kPPitch]
  float* red = reinterpret_cast<float*>(ps + R * S::kPPitch);                // [R][G] maxima; sums behind them at the end

  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = warp / G, kg = warp % G;
  const int split = blockIdx.x % p.splits, q_tile = blockIdx.x / p.splits, hg = blockIdx.y, seq = blockIdx.z;
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
  const int32_t* pages = p.page_table + (int64_t)seq * p.table_pitch;
  const int chunks = p.lat_pitch / 8;                                        // 16-byte pieces of a row; the rest stays zero

  // query rows, and zeros behind the rows' ends (query and key tiles)
  for (int r = warp; r < R; r += 8) {
    const int tok = r / nh, hd = r - tok * nh;
    const bf16* src = q_lat + ((int64_t)(start + tok0 + (r < rows ? tok : 0)) * p.heads + h0 + (r < rows ? hd : 0)) * p.lat_pitch;
    for (int c = lane; c < chunks; c += 32) cp_async16(sm_addr(qs + r * ld + 8 * c), src + 8 * c, r < rows);
    for (int c = chunks * 8 + lane; c < d16; c += 32) qs[r * ld + c] = __float2bfloat16_rn(0.0f);
  }
  for (int r = warp; r < 2 * NK; r += 8)
    for (int c = chunks * 8 + lane; c < d16; c += 32) ks[r * ld + c] = __float2bfloat16_rn(0.0f);

  auto load_tile = [&](int tile, int buf) {
    const int k0 = key_lo + tile * NK;
    int page[NK / 8];
#pragma unroll
    for (int i = 0; i < NK / 8; ++i) {
      const int key = k0 + warp + 8 * i;
      page[i] = key < key_hi ? __ldg(pages + key / kPage) : -1;
    }
#pragma unroll
    for (int i = 0; i < NK / 8; ++i) {
      const int r = warp + 8 * i, key = k0 + r;
      const bool ok = page[i] >= 0;
      const bf16* src = cache + ((int64_t)(ok ? page[i] : 0) * kPage + key % kPage) * p.lat_pitch;
      const unsigned dst = sm_addr(ks + (buf * NK + r) * ld);
      for (int c = lane; c < chunks; c += 32) cp_async16(dst + 16 * c, src + 8 * c, ok);
    }
  };
  if (tile0 < tile1) load_tile(tile0, 0);
  cp_async_commit();

  // this lane's two accumulator rows and the keys they may see
  int vis_lo[2], vis_hi[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = rg * 16 + (lane >> 2) + 8 * i;
    const int pos = pos0 + r / nh;
    vis_hi[i] = r < rows ? pos : -1;
    vis_lo[i] = p.window > 0 ? pos - p.window + 1 : 0;
  }
  float acc[NC16][2][4];
#pragma unroll
  for (int i = 0; i < NC16; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[i][j][k] = 0.0f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
  const int c16 = (p.kv_rank + 15) / 16, c_per = (c16 + G - 1) / G;          // 16-column pieces of the output, per column group
  const int c_lo = kg * c_per, c_n = max(0, min(c_per, c16 - c_lo));

  for (int tile = tile0; tile < tile1; ++tile) {
    const int buf = (tile - tile0) & 1;
    const bf16* kt = ks + buf * NK * ld;
    cp_async_wait<0>();
    __syncthreads();                                                         // tile arrived; the other buffer is free
    if (tile + 1 < tile1) load_tile(tile + 1, buf ^ 1);
    cp_async_commit();
    // scores: 16 rows x KW keys per warp, two accumulator sets to shorten the dependency chain
    float s[KT][4], s2[KT][4];
#pragma unroll
    for (int i = 0; i < KT; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) s[i][k] = s2[i][k] = 0.0f;
    const unsigned qa = sm_addr(qs + (rg * 16 + (lane & 15)) * ld + (lane >> 4) * 8);
    const unsigned kb4 = sm_addr(kt + (kg * KW + (lane & 7) + ((lane >> 4) << 3)) * ld + ((lane >> 3) & 1) * 8);
    const unsigned kb2 = sm_addr(kt + (kg * KW + (lane & 7)) * ld + ((lane >> 3) & 1) * 8);
    auto score_step = [&](int k, float (&dst)[KT][4]) {
      unsigned a[4];
      ldsm_x4(a, qa + 2 * k);
      if (KT == 1) {
        unsigned b0, b1;
        ldsm_x2(b0, b1, kb2 + 2 * k);
        mma_bf16(dst[0], a, b0, b1);
      } else {
#pragma unroll
        for (int i = 0; i + 1 < KT; i += 2) {
          unsigned b[4];
          ldsm_x4(b, kb4 + (unsigned)(i * 8 * ld * 2) + 2 * k);
          mma_bf16(dst[i], a, b[0], b[1]);
          mma_bf16(dst[i + 1 < KT ? i + 1 : i], a, b[2], b[3]);
        }
      }
    };
    int k = 0;
#pragma unroll 2
    for (; k + 16 < d16; k += 32) {
      score_step(k, s);
      score_step(k + 16, s2);
    }
    if (k < d16) score_step(k, s);
    // mask, scale, row maxima
    const int key0 = key_lo + tile * NK + kg * KW + 2 * (lane & 3);
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < KT; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int key = key0 + 8 * i + (j & 1), r = j >> 1;
        const float v = (key <= vis_hi[r] && key >= vis_lo[r]) ? (s[i][j] + s2[i][j]) * p.scale2 : -INFINITY;
        s[i][j] = v;
        mx[r] = fmaxf(mx[r], v);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(FULL_MASK, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(FULL_MASK, mx[r], 2));
      if ((lane & 3) == 0) red[(rg * 16 + (lane >> 2) + 8 * r) * G + kg] = mx[r];
    }
    __syncthreads();
    float alpha[2], mu[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mn = m[r];
#pragma unroll
      for (int g = 0; g < G; ++g) mn = fmaxf(mn, red[(rg * 16 + (lane >> 2) + 8 * r) * G + g]);
      mu[r] = mn == -INFINITY ? 0.0f : mn;                                   // no visible key so far: every weight is 0
      alpha[r] = exp2f(m[r] - mu[r]);
      m[r] = mn;
      l[r] *= alpha[r];
    }
#pragma unroll
    for (int i = 0; i < KT; ++i) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s[i][j] = exp2f(s[i][j] - mu[j >> 1]);
        l[j >> 1] += s[i][j];
      }
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<unsigned*>(ps + (rg * 16 + (lane >> 2) + 8 * r) * S::kPPitch + kg * KW + 8 * i + 2 * (lane & 3)) =
            f32_to_bf16x2(s[i][2 * r], s[i][2 * r + 1]);
    }
    __syncthreads();
    // output: 16 rows x this warp's columns
#pragma unroll
    for (int i = 0; i < NC16; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        acc[i][j][0] *= alpha[0]; acc[i][j][1] *= alpha[0];
        acc[i][j][2] *= alpha[1]; acc[i][j][3] *= alpha[1];
      }
    const unsigned pa = sm_addr(ps + (rg * 16 + (lane & 15)) * S::kPPitch + (lane >> 4) * 8);
    const unsigned vb = sm_addr(kt + (lane & 15) * ld + c_lo * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int kk = 0; kk < NK; kk += 16) {
      unsigned a[4];
      ldsm_x4(a, pa + 2 * kk);
#pragma unroll
      for (int i = 0; i < NC16; ++i) {
        if (i < c_n) {
          unsigned b[4];
          ldsm_x4_t(b, vb + (unsigned)(kk * ld * 2) + 32 * i);
          mma_bf16(acc[i][0], a, b[0], b[1]);
          mma_bf16(acc[i][1], a, b[2], b[3]);
        }
      }
    }
  }
  cp_async_wait<0>();
  // row sums over the key groups
  float* sums = red + R * G;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(FULL_MASK, l[r], 1);
    l[r] += __shfl_xor_sync(FULL_MASK, l[r], 2);
    if ((lane & 3) == 0) sums[(rg * 16 + (lane >> 2) + 8 * r) * G + kg] = l[r];
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = rg * 16 + (lane >> 2) + 8 * r;
    if (row >= rows) continue;
    float sum = 0.0f;
#pragma unroll
    for (int g = 0; g < G; ++g) sum += sums[row * G + g];
    const int tok = row / nh, hd = h0 + row - tok * nh;
    const int64_t gr = (int64_t)(start + tok0 + tok) * p.heads + hd;
    if (p.splits == 1) {
      const float sink2 = __ldg(p.sink + hd) * kLog2e, mf = fmaxf(m[r], sink2);
      const float inv = exp2f(m[r] - mf) / (sum * exp2f(m[r] - mf) + exp2f(sink2 - mf));
      bf16* dst = out + gr * p.out_pitch;
#pragma unroll
      for (int i = 0; i < NC16; ++i)
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
        ml[0] = m[r];
        ml[1] = sum;
      }
#pragma unroll
      for (int i = 0; i < NC16; ++i)
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
struct AttnPlan { int mt, nk, nc16; };      // mt = 0: the plain kernel

static AttnPlan plan_attn(int max_q, int heads, int kv_rank, int rot_dim) {
  const int d16 = (kv_rank + rot_dim + 15) & ~15, c16 = (kv_rank + 15) / 16;
  const size_t limit = 227 * 1024;
  const int64_t rows = (int64_t)max_q * heads;
  const int want = rows <= 16 ? 1 : (rows <= 32 ? 2 : 4);
  for (int mt = want; mt >= 1; mt >>= 1) {
    const int per = (c16 * mt + 7) / 8;
    if (mt == 4 && per <= 16) {
      const int nc = per <= 4 ? 4 : (per <= 8 ? 8 : 16);
      if (AttnShape<4, 64>::smem(d16) <= limit) return {4, 64, nc};
      if (AttnShape<4, 32>::smem(d16) <= limit) return {4, 32, nc};
    }
    if (mt == 2 && per <= 8) {
      const int nc = per <= 4 ? 4 : 8;
      if (AttnShape<2, 64>::smem(d16) <= limit) return {2, 64, nc};
      if (AttnShape<2, 32>::smem(d16) <= limit) return {2, 32, nc};
    }
    if (mt == 1 && per <= 8 && AttnShape<1, 64>::smem(d16) <= limit) return {1, 64, per <= 4 ? 4 : 8};
  }
  return {0, 0, 0};
}

static int attn_sm_count() {
  static int n = 0;
  if (n == 0) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
  }
  return n;
}

template <int MT, int NK, int NC16>
static int launch_mma(const AttnParams& p, const bf16* q, const bf16* cache, bf16* out, dim3 grid, int d16, cudaStream_t st) {
  const size_t smem = AttnShape<MT, NK>::smem(d16);
  cudaError_t e = cudaFuncSetAttribute(latent_attn_mma_kernel<MT, NK, NC16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "latent_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  launch_pdl(latent_attn_mma_kernel<MT, NK, NC16>, grid, dim3(256), smem, st, p, q, cache, out);
  return check_launch("latent_attn");
}

static int tiles_for(int max_q, int max_kv, int window, int tokens_per_cta, int nk) {
  int64_t span = max_kv;
  if (window > 0 && span > (int64_t)window + tokens_per_cta - 1) span = (int64_t)window + tokens_per_cta - 1;
  return (int)((span + nk - 1) / nk);
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
  const int tiles = tiles_for(max_q, max_kv, window, tpc, pl.nk);
  int64_t splits = attn_sm_count() / (ctas > 0 ? ctas : 1);
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
                          ? plan_attn(max_q, heads, kv_rank, rot_dim) : AttnPlan{0, 0, 0};
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
#define B200_ATTN_CASE(MT_, NK_, NC_) \
  if (pl.mt == MT_ && pl.nk == NK_ && pl.nc16 == NC_) rc = launch_mma<MT_, NK_, NC_>(p, q, kc, o, grid, d16, st);
  B200_ATTN_CASE(1, 64, 4)
  B200_ATTN_CASE(1, 64, 8)
  B200_ATTN_CASE(2, 64, 4)
  B200_ATTN_CASE(2, 64, 8)
  B200_ATTN_CASE(2, 32, 4)
  B200_ATTN_CASE(2, 32, 8)
  B200_ATTN_CASE(4, 64, 4)
  B200_ATTN_CASE(4, 64, 8)
  B200_ATTN_CASE(4, 64, 16)
  B200_ATTN_CASE(4, 32, 4)
  B200_ATTN_CASE(4, 32, 8)
  B200_ATTN_CASE(4, 32, 16)
#undef B200_ATTN_CASE
  if (rc != B200_OK || key_splits == 1) return rc;
  launch_pdl(latent_merge_kernel, dim3((unsigned)(tokens * heads)), dim3(128), 0, st, p, o);
  return check_launch("latent_attn (merge)");
}
