// Attention of grouped query heads over paged keys and values (16-token pages, heads / kv_heads query heads per key head),
// causal, with an optional window.
//
// grouped_prepare_kernel   between the projections and the scores: RMS norm of all of q and of all of k (before the split
//                          into heads), cache store; one CTA per token.
// grouped_attn_mma_kernel  bf16, prompts and decode.  The query heads of one key head are packed into the rows of a tile, so
//                          every key is read once for all of them.  Tiles of 64 keys come by cp.async, two in flight; scores
//                          and output on mma.sync with the softmax weights kept in registers between the two products.
//                          Prompts: each of 4 warps owns 16 rows and sees all keys.  Decode: all warps own the same (up to)
//                          16 rows, each takes 16 of a tile's 64 keys, and they meet once at the end; long key ranges of
//                          small batches are split over CTAs and merged by grouped_merge_kernel.
// grouped_attn_kernel      any size, any type, one CTA per (token, head); the 32-bit path.
// Scores, softmax and accumulators are fp32.
#include "float_common.cuh"
#include "umma.cuh"

namespace b200 {

constexpr int kGaPage = 16;
constexpr int kGaTile = 64;                // keys per tile
constexpr int kGaWarps = 4;
constexpr float kGaLog2e = 1.4426950408889634f;

// ---------------------------------------------------------------------------------------------------
struct GroupedPrepare {
  const float* y;
  int splits;
  int64_t split_stride, y_pitch, q_col, k_col, v_col;
  const float *q_norm, *k_norm;            // nullable: no norm
  float eps;
  const int32_t* out_loc;
  int heads, kv_heads, dim, vdim, dim_pitch, vdim_pitch;
  int64_t cache_rows;
};

template <typename T>
__global__ void __launch_bounds__(256)
grouped_prepare_kernel(const GroupedPrepare p, T* __restrict__ q, T* __restrict__ k_cache, T* __restrict__ v_cache) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const float* row = p.y + t * p.y_pitch;
  const int64_t loc = p.out_loc[t];
  const bool stores = loc >= 0 && loc < p.cache_rows;
  auto part = [&](int64_t col, int heads, int size, int pitch, const float* gain, T* dst) {
    const int n = heads * size;
    float inv = 1.0f;
    if (gain) {
      float ss = 0.0f;
      for (int i = threadIdx.x; i < n; i += 256) {
        const float v = part_sum(row + col + i, p.splits, p.split_stride);
        ss = fmaf(v, v, ss);
      }
      inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + p.eps);
    }
    if (!dst) return;
    for (int i = threadIdx.x; i < heads * pitch; i += 256) {
      const int h = i / pitch, e = i - h * pitch;
      float v = 0.0f;
      if (e < size) {
        v = part_sum(row + col + h * size + e, p.splits, p.split_stride) * inv;
        if (gain) v *= gain[h * size + e];
      }
      dst[i] = from_f32<T>(v);
    }
  };
  part(p.q_col, p.heads, p.dim, p.dim_pitch, p.q_norm, q + t * p.heads * p.dim_pitch);
  part(p.k_col, p.kv_heads, p.dim, p.dim_pitch, p.k_norm, stores ? k_cache + loc * p.kv_heads * p.dim_pitch : nullptr);
  part(p.v_col, p.kv_heads, p.vdim, p.vdim_pitch, nullptr, stores ? v_cache + loc * p.kv_heads * p.vdim_pitch : nullptr);
}

// ---------------------------------------------------------------------------------------------------
struct GroupedAttn {
  const int32_t* page_table;
  int64_t table_pitch;
  const int32_t *kv_lens, *seq_start;
  int64_t tokens;
  int heads, kv_heads, dim, vdim, dim_pitch, vdim_pitch, window;
  int64_t out_pitch;
  float scale2;                            // scale * log2(e)
  int splits;
  float* ws;                               // splits > 1: [splits][tokens * heads][vdim], then [splits][tokens * heads][2]
  int heads_per_cta, head_groups, tokens_per_cta;
};

__device__ __forceinline__ int ga_first_key(int pos, int window) { return window > 0 ? max(pos - window + 1, 0) : 0; }

template <typename T>
__global__ void __launch_bounds__(128)
grouped_attn_kernel(const GroupedAttn p, const T* __restrict__ q_in, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                    T* __restrict__ out, int batch) {
  extern __shared__ float sm[];
  pdl_launch_dependents();
  pdl_wait();
  float* q = sm;                           // [dim]
  float* o = q + p.dim;                    // [vdim]
  float* sc = o + p.vdim;                  // [128]
  float* red = sc + 128;                   // [8]
  const int64_t t = blockIdx.x;
  const int h = blockIdx.y, kvh = h / (p.heads / p.kv_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int seq = (int)t, first = (int)t, count = 1;
  if (p.seq_start) {
    int lo = 0, hi = batch;                // the sequence whose range holds token t
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.seq_start[mid] <= t) lo = mid; else hi = mid;
    }
    seq = lo; first = p.seq_start[seq]; count = p.seq_start[seq + 1] - first;
  }
  const int pos = p.kv_lens[seq] - count + (int)(t - first);
  const int32_t* pages = p.page_table + (int64_t)seq * p.table_pitch;
  auto row_of = [&](int key) { return ((int64_t)pages[key / kGaPage] * kGaPage + key % kGaPage) * p.kv_heads + kvh; };
  const T* qs = q_in + (t * p.heads + h) * p.dim_pitch;
  for (int i = threadIdx.x; i < p.dim; i += 128) q[i] = to_f32(qs[i]);
  for (int i = threadIdx.x; i < p.vdim; i += 128) o[i] = 0.0f;
  float m = -INFINITY, l = 0.0f;
  __syncthreads();
  for (int k0 = ga_first_key(pos, p.window); k0 <= pos; k0 += 128) {
    const int n = min(128, pos + 1 - k0);
    for (int j = warp; j < n; j += 4) {
      const T* row = k_cache + row_of(k0 + j) * p.dim_pitch;
      float s = 0.0f;
      for (int i = lane; i < p.dim; i += 32) s = fmaf(q[i], to_f32(row[i]), s);
      s = warp_sum(s);
      if (lane == 0) sc[j] = s * p.scale2;
    }
    __syncthreads();
    const float v = (int)threadIdx.x < n ? sc[threadIdx.x] : -INFINITY;
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
    for (int i = threadIdx.x; i < p.vdim; i += 128) {
      float acc = o[i] * alpha;
      for (int j = 0; j < n; ++j) acc = fmaf(sc[j], to_f32(v_cache[row_of(k0 + j) * p.vdim_pitch + i]), acc);
      o[i] = acc;
    }
    __syncthreads();
  }
  T* dst = out + t * p.out_pitch + (int64_t)h * p.vdim;
  for (int i = threadIdx.x; i < p.vdim; i += 128) dst[i] = from_f32<T>(o[i] / l);
}

// ---------------------------------------------------------------------------------------------------
__device__ __forceinline__ void ga_ldsm(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ga_ldsm_t(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ga_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ga_exp2(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}

__host__ __device__ constexpr int ga_ld(int n) { return ((n + 15) & ~15) + 8; }         // shared row pitch: conflict-free ldmatrix

// D16: most 16-column pieces of a key or value; FULL: exactly that many.  DECODE: every warp has the same 16 rows and a quarter
// of each key tile.
template <int D16, bool DECODE, bool FULL>
__global__ void __launch_bounds__(kGaWarps * 32)
grouped_attn_mma_kernel(const GroupedAttn p, const bf16* __restrict__ q_in, const bf16* __restrict__ k_cache,
                        const bf16* __restrict__ v_cache, bf16* __restrict__ out) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  constexpr int NT = kGaTile, THREADS = kGaWarps * 32;
  constexpr int KW = DECODE ? NT / kGaWarps : NT;                      // keys of a tile per warp
  const int ldk = FULL ? ga_ld(16 * D16) : ga_ld(p.dim), ldv = FULL ? ga_ld(16 * D16) : ga_ld(p.vdim);
  const int k16 = (p.dim + 15) >> 4, c16 = (p.vdim + 15) >> 4;
  bf16* ks = reinterpret_cast<bf16*>(smem_raw);                        // [2][NT][ldk]
  bf16* vs = ks + 2 * NT * ldk;                                        // [2][NT][ldv]

  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x % p.splits, q_tile = blockIdx.x / p.splits, seq = blockIdx.z;
  const int kvh = blockIdx.y / p.head_groups, hg = blockIdx.y % p.head_groups, per = p.heads / p.kv_heads;
  for (int r = warp; r < 2 * NT; r += kGaWarps) {                      // columns behind a row's copied part stay zero
    for (int c = p.dim_pitch + lane; c < ldk; c += 32) ks[r * ldk + c] = __float2bfloat16_rn(0.0f);
    for (int c = p.vdim_pitch + lane; c < ldv; c += 32) vs[r * ldv + c] = __float2bfloat16_rn(0.0f);
  }
  pdl_wait();
  const int start = p.seq_start ? p.seq_start[seq] : seq;
  const int count = p.seq_start ? p.seq_start[seq + 1] - start : 1;
  const int tok0 = q_tile * p.tokens_per_cta;
  if (tok0 >= count) return;
  const int ntok = min(p.tokens_per_cta, count - tok0);
  const int h0 = kvh * per + hg * p.heads_per_cta, nh = min(p.heads_per_cta, per - hg * p.heads_per_cta);
  const int rows = ntok * nh;
  const int pos0 = p.kv_lens[seq] - count + tok0;
  const int key_lo = ga_first_key(pos0, p.window), key_hi = pos0 + ntok;      // keys that some row sees
  const int base = key_lo & ~(kGaPage - 1);
  const int all_tiles = (key_hi - base + NT - 1) / NT, per_split = (all_tiles + p.splits - 1) / p.splits;
  const int tile0 = split * per_split, tile1 = min(all_tiles, tile0 + per_split);
  const int32_t* pages = p.page_table + (int64_t)seq * p.table_pitch;

  // Each warp copies one of a tile's four pages, a 16-byte piece of the key or value of all 16 rows per lane; keys outside
  // [key_lo, key_hi) become zeros.  The page id is looked up a tile ahead.
  static_assert(NT == kGaWarps * kGaPage, "a page per warp");
  const int ck = p.dim_pitch / 8, chunks = ck + p.vdim_pitch / 8, last_page = (key_hi - 1) / kGaPage;
  int page = 0;
  auto look_up = [&](int tile) { page = __ldg(pages + min((base + tile * NT) / kGaPage + warp, last_page)); };
  auto issue = [&](int tile) {                   // needs look_up(tile)
    const int buf = (tile - tile0) & 1, r0 = warp * kGaPage, k0 = base + tile * NT + r0;
    const bool all = k0 >= key_lo && k0 + kGaPage <= key_hi;
    for (int c = lane; c < chunks; c += 32) {
      const bool is_k = c < ck;
      const int pitch = is_k ? p.dim_pitch : p.vdim_pitch, col = (is_k ? c : c - ck) * 8, ld = is_k ? ldk : ldv;
      const bf16* src = (is_k ? k_cache : v_cache) + ((int64_t)page * kGaPage * p.kv_heads + kvh) * pitch + col;
      unsigned dst = smem_u32((is_k ? ks : vs) + (buf * NT + r0) * ld + col);
      const int64_t step = (int64_t)p.kv_heads * pitch;
      if (all) {
#pragma unroll
        for (int r = 0; r < kGaPage; ++r) {
          cp_async16(dst, src);
          src += step;
          dst += 2 * ld;
        }
      } else {
        for (int r = 0; r < kGaPage; ++r) {
          const int live = k0 + r >= key_lo && k0 + r < key_hi ? 16 : 0;
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live) : "memory");
          src += step;
          dst += 2 * ld;
        }
      }
    }
    if (tile + 1 < tile1) look_up(tile + 1);
  };
  if (tile0 < tile1) {
    look_up(tile0);
    issue(tile0);
  }
  cp_async_commit();

  const int row_base = DECODE ? 0 : warp * 16;
  unsigned qf[D16][4];
  int vis_hi[2], vis_lo[2];
  {
    const bf16* src[2];
    bool live[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = row_base + (lane >> 2) + 8 * i, tok = r / nh;
      live[i] = r < rows;
      const int pos = pos0 + tok;
      vis_hi[i] = live[i] ? pos : -1;
      vis_lo[i] = p.window > 0 ? pos - p.window + 1 : 0;
      src[i] = q_in + ((int64_t)(start + tok0 + (live[i] ? tok : 0)) * p.heads + h0 + (live[i] ? r - tok * nh : 0)) * p.dim_pitch;
    }
#pragma unroll
    for (int i = 0; i < D16; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = i * 16 + 8 * (j >> 1) + 2 * (lane & 3);
        qf[i][j] = (live[j & 1] && col < p.dim_pitch) ? __ldg(reinterpret_cast<const unsigned*>(src[j & 1] + col)) : 0u;
      }
  }
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
  float acc[D16][2][4];
#pragma unroll
  for (int i = 0; i < D16; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[i][j][k] = 0.0f;
  const int key_off = DECODE ? warp * KW : 0;
  const unsigned k_lane = (key_off + (lane & 7) + ((lane >> 4) << 3)) * ldk + ((lane >> 3) & 1) * 8;
  const unsigned v_lane = (key_off + (lane & 15)) * ldv + (lane >> 4) * 8;
  // first and last key that this warp's rows see: tiles outside are skipped
  const int warp_lo = DECODE ? key_lo : ga_first_key(pos0 + min(row_base, rows - 1) / nh, p.window);
  const int warp_hi = DECODE ? key_hi : pos0 + min(row_base + 15, rows - 1) / nh + 1;
  const bool warp_live = row_base < rows;
  // keys [all_lo, all_hi) are seen by every row (rows behind the last one do not matter)
  const int all_lo = ga_first_key(pos0 + (DECODE ? ntok - 1 : min(row_base + 15, rows - 1) / nh), p.window);
  const int all_hi = pos0 + (DECODE ? 0 : min(row_base, rows - 1) / nh) + 1;

  for (int tile = tile0; tile < tile1; ++tile) {
    const int buf = (tile - tile0) & 1;
    if (tile + 1 < tile1) issue(tile + 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const int key0 = base + tile * NT + key_off;
    if (warp_live && key0 < warp_hi && key0 + KW > warp_lo) {
      float s[KW / 8][4];
#pragma unroll
      for (int i = 0; i < KW / 8; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) s[i][k] = 0.0f;
      const unsigned kb = smem_u32(ks + buf * NT * ldk + k_lane);
#pragma unroll
      for (int i = 0; i < D16; ++i) {
        if (FULL || i < k16) {
#pragma unroll
          for (int n = 0; n < KW / 16; ++n) {
            unsigned b[4];
            ga_ldsm(b, kb + (unsigned)(n * 16 * ldk * 2) + 32 * i);
            ga_mma(s[2 * n], qf[i], b[0], b[1]);
            ga_mma(s[2 * n + 1], qf[i], b[2], b[3]);
          }
        }
      }
      float mn[2] = {m[0], m[1]};
      if (key0 >= all_lo && key0 + KW <= all_hi) {
#pragma unroll
        for (int i = 0; i < KW / 8; ++i)
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            s[i][k] *= p.scale2;
            mn[k >> 1] = fmaxf(mn[k >> 1], s[i][k]);
          }
      } else {
#pragma unroll
        for (int i = 0; i < KW / 8; ++i)
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const int key = key0 + 8 * i + 2 * (lane & 3) + (k & 1), r = k >> 1;
            s[i][k] = (key <= vis_hi[r] && key >= vis_lo[r]) ? s[i][k] * p.scale2 : -INFINITY;
            mn[r] = fmaxf(mn[r], s[i][k]);
          }
      }
      float alpha[2], mu[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mn[r] = fmaxf(mn[r], __shfl_xor_sync(FULL_MASK, mn[r], 1));
        mn[r] = fmaxf(mn[r], __shfl_xor_sync(FULL_MASK, mn[r], 2));
        mu[r] = mn[r] == -INFINITY ? 0.0f : mn[r];               // no visible key so far: every weight is 0
        alpha[r] = ga_exp2(m[r] - mu[r]);
        m[r] = mn[r];
        l[r] *= alpha[r];
      }
#pragma unroll
      for (int i = 0; i < KW / 8; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          s[i][k] = ga_exp2(s[i][k] - mu[k >> 1]);
          l[k >> 1] += s[i][k];
        }
      if (__any_sync(FULL_MASK, alpha[0] != 1.0f || alpha[1] != 1.0f)) {
#pragma unroll
        for (int i = 0; i < D16; ++i)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            acc[i][j][0] *= alpha[0]; acc[i][j][1] *= alpha[0];
            acc[i][j][2] *= alpha[1]; acc[i][j][3] *= alpha[1];
          }
      }
      const unsigned vb = smem_u32(vs + buf * NT * ldv + v_lane);
#pragma unroll
      for (int kk = 0; kk < KW / 16; ++kk) {
        const unsigned a[4] = {f32_to_bf16x2(s[2 * kk][0], s[2 * kk][1]), f32_to_bf16x2(s[2 * kk][2], s[2 * kk][3]),
                               f32_to_bf16x2(s[2 * kk + 1][0], s[2 * kk + 1][1]), f32_to_bf16x2(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
        for (int i = 0; i < D16; ++i) {
          if (FULL || i < c16) {
            unsigned b[4];
            ga_ldsm_t(b, vb + (unsigned)(kk * 16 * ldv * 2) + 32 * i);
            ga_mma(acc[i][0], a, b[0], b[1]);
            ga_mma(acc[i][1], a, b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();                                             // the buffer may be refilled
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(FULL_MASK, l[r], 1);
    l[r] += __shfl_xor_sync(FULL_MASK, l[r], 2);
  }
  cp_async_wait<0>();
  if constexpr (DECODE) {
    // the warps' parts: maxima and sums first, then the outputs added through shared memory
    float* ml = reinterpret_cast<float*>(smem_raw);              // [warps][16][2]
    float* os = ml + kGaWarps * 32;                              // [warps][16][vdim + 4]
    const int lo = p.vdim + 4;
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = (lane >> 2) + 8 * r;
      if ((lane & 3) == 0) {
        ml[(warp * 16 + row) * 2] = m[r];
        ml[(warp * 16 + row) * 2 + 1] = l[r];
      }
#pragma unroll
      for (int i = 0; i < D16; ++i)
        if (i < c16) {
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int col = i * 16 + 8 * j + 2 * (lane & 3);
            if (col < p.vdim) os[(warp * 16 + row) * lo + col] = acc[i][j][2 * r];
            if (col + 1 < p.vdim) os[(warp * 16 + row) * lo + col + 1] = acc[i][j][2 * r + 1];
          }
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < rows * p.vdim; i += THREADS) {
      const int row = i / p.vdim, col = i - row * p.vdim;
      float mx = -INFINITY;
#pragma unroll
      for (int w = 0; w < kGaWarps; ++w) mx = fmaxf(mx, ml[(w * 16 + row) * 2]);
      float v = 0.0f, sum = 0.0f;
#pragma unroll
      for (int w = 0; w < kGaWarps; ++w) {
        const float f = mx == -INFINITY ? 0.0f : exp2f(ml[(w * 16 + row) * 2] - mx);
        sum = fmaf(f, ml[(w * 16 + row) * 2 + 1], sum);
        v = fmaf(f, os[(w * 16 + row) * lo + col], v);
      }
      const int tok = row / nh, hd = h0 + row - tok * nh;
      const int64_t tk = start + tok0 + tok;
      if (p.splits == 1) {
        out[tk * p.out_pitch + (int64_t)hd * p.vdim + col] = __float2bfloat16_rn(v / sum);
      } else {
        const int64_t all = p.tokens * p.heads, gr = tk * p.heads + hd;
        p.ws[((int64_t)split * all + gr) * p.vdim + col] = v;
        if (col == 0) {
          float* e = p.ws + (int64_t)p.splits * all * p.vdim + ((int64_t)split * all + gr) * 2;
          e[0] = mx;
          e[1] = sum;
        }
      }
    }
  } else {
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = row_base + (lane >> 2) + 8 * r;
    if (row >= rows) continue;
    const int tok = row / nh, hd = h0 + row - tok * nh;
    const float inv = 1.0f / l[r];
    bf16* dst = out + (int64_t)(start + tok0 + tok) * p.out_pitch + (int64_t)hd * p.vdim;
    const bool pair = ((reinterpret_cast<uintptr_t>(dst) & 3) == 0);
#pragma unroll
    for (int i = 0; i < D16; ++i)
      if (FULL || i < c16) {
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int col = i * 16 + 8 * j + 2 * (lane & 3);
          const float a = acc[i][j][2 * r] * inv, b = acc[i][j][2 * r + 1] * inv;
          if (pair && col + 1 < p.vdim) {
            *reinterpret_cast<unsigned*>(dst + col) = f32_to_bf16x2(a, b);
          } else {
            if (col < p.vdim) dst[col] = __float2bfloat16_rn(a);
            if (col + 1 < p.vdim) dst[col + 1] = __float2bfloat16_rn(b);
          }
        }
      }
  }
  }
}

// Parts of the key range of one (token, head) row merged.
__global__ void __launch_bounds__(128)
grouped_merge_kernel(const GroupedAttn p, bf16* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t gr = blockIdx.x, all = p.tokens * p.heads;
  const float* ml = p.ws + (int64_t)p.splits * all * p.vdim;
  float m = -INFINITY;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ml[((int64_t)s * all + gr) * 2]);
  float sum = 0.0f;
  for (int s = 0; s < p.splits; ++s) {
    const float* e = ml + ((int64_t)s * all + gr) * 2;
    sum += e[1] * exp2f(e[0] - m);
  }
  const float inv = 1.0f / sum;
  for (int c = threadIdx.x; c < p.vdim; c += 128) {
    float v = 0.0f;
    for (int s = 0; s < p.splits; ++s) v = fmaf(exp2f(ml[((int64_t)s * all + gr) * 2] - m), p.ws[((int64_t)s * all + gr) * p.vdim + c], v);
    out[(gr / p.heads) * p.out_pitch + (gr % p.heads) * p.vdim + c] = __float2bfloat16_rn(v * inv);
  }
}

// ----------------------------------------------------------------------------- host side
static size_t ga_smem(int dim, int vdim, bool decode) {
  const size_t tiles = (size_t)2 * kGaTile * (ga_ld(dim) + ga_ld(vdim)) * 2;
  const size_t merge = (size_t)kGaWarps * (32 + 16 * (vdim + 4)) * 4;
  return decode && merge > tiles ? merge : tiles;
}
static bool ga_decode_form(int max_q, int heads, int kv_heads) { return max_q == 1 && heads / kv_heads > 0; }
static int ga_rows(bool decode) { return decode ? 16 : 16 * kGaWarps; }

template <int D16, bool DECODE, bool FULL>
static int launch_ga(const GroupedAttn& p, const bf16* q, const bf16* k, const bf16* v, bf16* out, dim3 grid, size_t smem, cudaStream_t st) {
  cudaError_t e = cudaFuncSetAttribute(grouped_attn_mma_kernel<D16, DECODE, FULL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "grouped_attn: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  launch_pdl(grouped_attn_mma_kernel<D16, DECODE, FULL>, grid, dim3(kGaWarps * 32), smem, st, p, q, k, v, out);
  return check_launch("grouped_attn");
}
static bool ga_mma_fits(int dim, int vdim, int dtype) {
  return dtype == B200F_BF16 && dim <= 256 && vdim <= 256 && ga_smem(dim, vdim, true) <= 227 * 1024;
}

}  // namespace b200

using namespace b200;

extern "C" int b200f_grouped_prepare(const float* y, int splits, int64_t split_stride, int64_t y_pitch, int64_t q_col,
                                     int64_t k_col, int64_t v_col, const float* q_norm, const float* k_norm, float eps,
                                     const int32_t* out_loc, void* q, void* k_cache, void* v_cache, int dtype, int64_t tokens,
                                     int heads, int kv_heads, int dim, int vdim, int dim_pitch, int vdim_pitch,
                                     int64_t cache_rows, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "grouped_prepare: dtype %d", dtype);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && splits >= 1 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0 &&
                   dim_pitch >= dim && vdim_pitch >= vdim && cache_rows >= 0 && q_col >= 0 && k_col >= 0 && v_col >= 0 &&
                   q_col + (int64_t)heads * dim <= y_pitch && k_col + (int64_t)kv_heads * dim <= y_pitch && v_col + (int64_t)kv_heads * vdim <= y_pitch,
               B200_E_SHAPE, "grouped_prepare: tokens=%lld heads=%d/%d dim=%d vdim=%d", (long long)tokens, heads, kv_heads, dim, vdim);
  if (tokens == 0) return B200_OK;
  B200_REQUIRE(y && out_loc && q && k_cache && v_cache, B200_E_NULL, "grouped_prepare: null pointer");
  GroupedPrepare p{y, splits, split_stride, y_pitch, q_col, k_col, v_col, q_norm, k_norm, eps, out_loc, heads, kv_heads, dim, vdim, dim_pitch,
                   vdim_pitch, cache_rows};
  if (dtype == B200F_BF16)
    launch_pdl(grouped_prepare_kernel<bf16>, dim3((unsigned)tokens), dim3(256), 0, (cudaStream_t)s, p, (bf16*)q, (bf16*)k_cache, (bf16*)v_cache);
  else
    launch_pdl(grouped_prepare_kernel<float>, dim3((unsigned)tokens), dim3(256), 0, (cudaStream_t)s, p, (float*)q, (float*)k_cache, (float*)v_cache);
  return check_launch("grouped_prepare");
}

extern "C" size_t b200f_grouped_attn_ws_floats(int64_t tokens, int heads, int vdim, int key_splits) {
  return key_splits > 1 ? (size_t)key_splits * (size_t)tokens * (size_t)heads * ((size_t)vdim + 2) : 0;
}

extern "C" int b200f_grouped_attn_splits(int64_t tokens, int batch, int max_q, int max_kv, int heads, int kv_heads, int dim,
                                         int vdim, int window, int dtype) {
  if (tokens <= 0 || batch <= 0 || kv_heads <= 0 || !ga_mma_fits(dim, vdim, dtype) || !ga_decode_form(max_q, heads, kv_heads)) return 1;
  const int per = heads / kv_heads, groups = (per + 15) / 16;
  const int64_t ctas = (int64_t)batch * kv_heads * groups;
  int64_t span = max_kv;
  if (window > 0 && span > (int64_t)window + kGaPage) span = (int64_t)window + kGaPage;
  const int64_t tiles = (span + kGaTile - 1) / kGaTile;
  int64_t splits = 4ll * sm_count() / (ctas > 0 ? ctas : 1);
  if (splits > tiles / 2) splits = tiles / 2;                    // a part keeps at least two key tiles
  return (int)(splits < 1 ? 1 : (splits > 32 ? 32 : splits));
}

extern "C" int b200f_grouped_attn(const void* q, const void* k_cache, const void* v_cache, const int32_t* page_table,
                                  int64_t table_pitch, const int32_t* kv_lens, const int32_t* seq_start, void* out, int dtype,
                                  int64_t tokens, int batch, int max_q, int heads, int kv_heads, int dim, int vdim,
                                  int dim_pitch, int vdim_pitch, int64_t out_pitch, int window, float scale, int key_splits,
                                  float* ws, int simple, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "grouped_attn: dtype %d", dtype);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && batch >= 0 && batch < 65536 && max_q > 0 && heads > 0 && heads < 65536 && kv_heads > 0 &&
                   heads % kv_heads == 0 && dim > 0 && vdim > 0 && dim_pitch >= dim && vdim_pitch >= vdim && out_pitch >= (int64_t)heads * vdim &&
                   window >= 0 && table_pitch > 0 && key_splits >= 1 && (seq_start || (tokens == batch && max_q == 1)),
               B200_E_SHAPE, "grouped_attn: tokens=%lld batch=%d heads=%d/%d dim=%d vdim=%d window=%d", (long long)tokens, batch, heads, kv_heads, dim, vdim, window);
  if (tokens == 0 || batch == 0) return B200_OK;
  B200_REQUIRE(q && k_cache && v_cache && page_table && kv_lens && out && (key_splits == 1 || ws), B200_E_NULL, "grouped_attn: null pointer");
  cudaStream_t st = (cudaStream_t)s;
  GroupedAttn p{page_table, table_pitch, kv_lens, seq_start, tokens, heads, kv_heads, dim, vdim, dim_pitch, vdim_pitch, window, out_pitch,
                scale * kGaLog2e, key_splits, ws, 1, 1, 1};
  const bool mma = !simple && ga_mma_fits(dim, vdim, dtype) && dim_pitch % 8 == 0 && vdim_pitch % 8 == 0 && dim_pitch < dim + 8 &&
                   vdim_pitch < vdim + 8 && aligned16(q) && aligned16(k_cache) && aligned16(v_cache);
  const bool decode = mma && ga_decode_form(max_q, heads, kv_heads);
  B200_REQUIRE(key_splits == 1 || decode, B200_E_UNSUPPORTED, "grouped_attn: key_splits=%d needs the decode form", key_splits);
  if (!mma) {
    const size_t smem = (size_t)(dim + vdim + 128 + 8) * sizeof(float);
    B200_REQUIRE(smem <= 48 * 1024, B200_E_UNSUPPORTED, "grouped_attn: heads of %d and %d values are too large", dim, vdim);
    const dim3 grid((unsigned)tokens, (unsigned)heads);
    if (dtype == B200F_BF16)
      launch_pdl(grouped_attn_kernel<bf16>, grid, dim3(128), smem, st, p, (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, (bf16*)out, batch);
    else
      launch_pdl(grouped_attn_kernel<float>, grid, dim3(128), smem, st, p, (const float*)q, (const float*)k_cache, (const float*)v_cache, (float*)out, batch);
    return check_launch("grouped_attn (plain)");
  }
  const int rows = ga_rows(decode), per = heads / kv_heads;
  p.heads_per_cta = per < rows ? per : rows;
  p.head_groups = (per + p.heads_per_cta - 1) / p.heads_per_cta;
  p.tokens_per_cta = decode ? 1 : rows / p.heads_per_cta;
  const int64_t q_tiles = (max_q + p.tokens_per_cta - 1) / p.tokens_per_cta;
  B200_REQUIRE(q_tiles * key_splits < (1ll << 31) && (int64_t)kv_heads * p.head_groups < 65536, B200_E_SHAPE, "grouped_attn: too many tiles");
  const dim3 grid((unsigned)(q_tiles * key_splits), (unsigned)(kv_heads * p.head_groups), (unsigned)batch);
  const size_t smem = ga_smem(dim, vdim, decode);
  const bf16 *qq = (const bf16*)q, *kk = (const bf16*)k_cache, *vv = (const bf16*)v_cache;
  bf16* o = (bf16*)out;
  const int big = dim > vdim ? dim : vdim;
  int rc;
#define B200_GA_CASE(D16_)                                                                                                                     \
  if (dim == 16 * D16_ && vdim == dim)                                                                                                        \
    rc = decode ? launch_ga<D16_, true, true>(p, qq, kk, vv, o, grid, smem, st) : launch_ga<D16_, false, true>(p, qq, kk, vv, o, grid, smem, st);   \
  else                                                                                                                                        \
    rc = decode ? launch_ga<D16_, true, false>(p, qq, kk, vv, o, grid, smem, st) : launch_ga<D16_, false, false>(p, qq, kk, vv, o, grid, smem, st);
  if (big <= 64) { B200_GA_CASE(4) }
  else if (big <= 128) { B200_GA_CASE(8) }
  else { B200_GA_CASE(16) }
#undef B200_GA_CASE
  if (rc != B200_OK || key_splits == 1) return rc;
  launch_pdl(grouped_merge_kernel, dim3((unsigned)(tokens * heads)), dim3(128), 0, st, p, o);
  return check_launch("grouped_attn (merge)");
}
