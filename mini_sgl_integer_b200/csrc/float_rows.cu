// Row kernels of the floating-point models: embedding (+ bigram row), the end of a sublayer (mean of two normed outputs,
// output norm, residual add, added vector, depth average, norm in front of the next linear), xIELU, gated SiLU, and the
// arg-max over fp32 logits.  Streams, norms and averages are fp32; the
// T-typed copies feed the next linear.
#include "float_common.cuh"

namespace b200 {

// ---------------------------------------------------------------------------------------------------
// Embedding: one CTA per token.  The thread that reads the stored previous token of a sequence (its first new token's
// CTA) also replaces it by the last new one, so no other CTA can see the new value too early.
// ---------------------------------------------------------------------------------------------------
struct EmbedParams {
  const int32_t *ids, *positions, *seq_ids, *seq_start, *slots;
  int32_t* prev_tokens;
  float* out;
  int width;
  int64_t vocab, buckets, mul_prev, mul_cur, out_t_pitch;
};

template <typename T>
__global__ void __launch_bounds__(128)
embed_bigram_kernel(const T* __restrict__ table, const T* __restrict__ bigram, T* __restrict__ out_t, const EmbedParams p) {
  __shared__ int64_t s_row[2];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t = blockIdx.x;
  if (threadIdx.x == 0) {
    const int64_t id = p.ids[t];
    s_row[0] = id >= 0 && id < p.vocab ? id : -1;
    if (bigram) {
      const int seq = p.seq_ids ? p.seq_ids[t] : (int)t;
      const int64_t first = p.seq_start ? p.seq_start[seq] : t;
      int64_t prev = -1;
      if (t == first) {
        const int slot = p.slots[seq];
        if (p.positions[t] > 0) prev = p.prev_tokens[slot];
        p.prev_tokens[slot] = p.seq_start ? p.ids[p.seq_start[seq + 1] - 1] : (int32_t)id;
      } else {
        prev = p.ids[t - 1];
      }
      int64_t row = p.buckets;
      if (p.positions[t] > 0) {
        row = (prev * p.mul_prev + id * p.mul_cur) % p.buckets;
        if (row < 0) row += p.buckets;
      }
      s_row[1] = row;
    }
  }
  __syncthreads();
  const int64_t r0 = s_row[0];
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    float v = r0 >= 0 ? to_f32(table[r0 * p.width + c]) : 0.0f;
    if (bigram) v += to_f32(bigram[s_row[1] * p.width + c]);
    p.out[t * p.width + c] = v;
    if (out_t) out_t[t * p.out_t_pitch + c] = from_f32<T>(v);
  }
}

// ---------------------------------------------------------------------------------------------------
// End of a sublayer, one CTA per token row held in registers: NV groups of VEC values per thread.
// ---------------------------------------------------------------------------------------------------
struct SublayerEnd {
  const float* y;
  int splits;
  int64_t split_stride;
  const float* y2;                   // nullable: the output is the mean of y normed with gain w1 and y2 normed with gain w2
  int splits2;
  int64_t split_stride2;
  const float *w1, *w2;
  const float *x_in, *norm_w;        // x_in nullable: zero
  const float* add;                  // nullable: a vector for every row
  float* x_out;
  const float* hist;
  int planes;
  int64_t plane_stride;
  const float* coef;
  float* hist_out;
  const float* final_w;
  int width;
  int64_t t_pitch;
  float eps;
};

template <int VEC>
struct Pack { float v[VEC]; };
template <int VEC>
__device__ __forceinline__ Pack<VEC> load_pack(const float* p) {
  Pack<VEC> r;
  if (VEC == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    r.v[0] = a.x; r.v[VEC > 1 ? 1 : 0] = a.y; r.v[VEC > 2 ? 2 : 0] = a.z; r.v[VEC > 3 ? 3 : 0] = a.w;
    if (VEC == 1) r.v[0] = a.x;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ void store_pack(float* p, const Pack<VEC>& a) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[VEC > 1 ? 1 : 0], a.v[VEC > 2 ? 2 : 0], a.v[VEC > 3 ? 3 : 0]);
  else *p = a.v[0];
}
template <int VEC>
__device__ __forceinline__ void store_pack(bf16* p, const Pack<VEC>& a) {
  if (VEC == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(f32_to_bf16x2(a.v[0], a.v[VEC > 1 ? 1 : 0]), f32_to_bf16x2(a.v[VEC > 2 ? 2 : 0], a.v[VEC > 3 ? 3 : 0]));
  } else {
    *p = __float2bfloat16_rn(a.v[0]);
  }
}

template <typename T, int VEC, int NV>
__global__ void sublayer_end_kernel(const SublayerEnd p, T* __restrict__ x_out_t) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const int64_t row = blockIdx.x;
  const int64_t base = row * p.width;
  pdl_wait();
  Pack<VEC> r[NV];
  int col[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) col[i] = (i * blockDim.x + threadIdx.x) * VEC;
  // the sum of a stack of parts and its sum of squares
  auto take = [&](const float* y, int splits, int64_t stride, Pack<VEC> (&a)[NV]) {
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (col[i] >= p.width) continue;
      a[i] = load_pack<VEC>(y + base + col[i]);
      for (int s = 1; s < splits; ++s) {
        const Pack<VEC> o = load_pack<VEC>(y + (int64_t)s * stride + base + col[i]);
#pragma unroll
        for (int k = 0; k < VEC; ++k) a[i].v[k] += o.v[k];
      }
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(a[i].v[k], a[i].v[k], ss);
    }
    return ss;
  };
  if (p.y) {
    float ss = take(p.y, p.splits, p.split_stride, r);
    if (p.y2) {
      Pack<VEC> r2[NV];
      const float ss2 = block_sum(take(p.y2, p.splits2, p.split_stride2, r2), scratch);
      const float i1 = 0.5f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.eps), i2 = 0.5f / sqrtf(ss2 / (float)p.width + p.eps);
      ss = 0.0f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (col[i] >= p.width) continue;
        const Pack<VEC> a = load_pack<VEC>(p.w1 + col[i]), b = load_pack<VEC>(p.w2 + col[i]);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          r[i].v[k] = fmaf(r[i].v[k] * i1, a.v[k], r2[i].v[k] * i2 * b.v[k]);
          ss = fmaf(r[i].v[k], r[i].v[k], ss);
        }
      }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)p.width + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (col[i] >= p.width) continue;
      Pack<VEC> x;
#pragma unroll
      for (int k = 0; k < VEC; ++k) x.v[k] = 0.0f;
      if (p.x_in) x = load_pack<VEC>(p.x_in + base + col[i]);
      const Pack<VEC> w = load_pack<VEC>(p.norm_w + col[i]);
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[i].v[k] = fmaf(r[i].v[k] * inv, w.v[k], x.v[k]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < p.width) r[i] = load_pack<VEC>(p.x_in + base + col[i]);
  }
  if (p.add) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (col[i] >= p.width) continue;
      const Pack<VEC> a = load_pack<VEC>(p.add + col[i]);
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[i].v[k] += a.v[k];
    }
  }
  if (p.coef) {
    const float c_new = p.coef[p.planes];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (col[i] >= p.width) continue;
      if (p.hist_out) store_pack<VEC>(p.hist_out + base + col[i], r[i]);
      Pack<VEC> a;
#pragma unroll
      for (int k = 0; k < VEC; ++k) a.v[k] = 0.0f;
      const float* h = p.hist + base + col[i];
      int j = 0;
      for (; j + 4 <= p.planes; j += 4) {          // four planes in flight
        Pack<VEC> b[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) b[u] = load_pack<VEC>(h + (int64_t)(j + u) * p.plane_stride);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float c = __ldg(p.coef + j + u);
#pragma unroll
          for (int k = 0; k < VEC; ++k) a.v[k] = fmaf(c, b[u].v[k], a.v[k]);
        }
      }
      for (; j < p.planes; ++j) {
        const Pack<VEC> b = load_pack<VEC>(h + (int64_t)j * p.plane_stride);
        const float c = __ldg(p.coef + j);
#pragma unroll
        for (int k = 0; k < VEC; ++k) a.v[k] = fmaf(c, b.v[k], a.v[k]);
      }
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[i].v[k] = fmaf(c_new, r[i].v[k], a.v[k]);
    }
  }
  if (p.x_out) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < p.width) store_pack<VEC>(p.x_out + base + col[i], r[i]);
  }
  if (p.final_w) {
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < p.width) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) ss = fmaf(r[i].v[k], r[i].v[k], ss);
      }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)p.width + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (col[i] >= p.width) continue;
      const Pack<VEC> w = load_pack<VEC>(p.final_w + col[i]);
#pragma unroll
      for (int k = 0; k < VEC; ++k) r[i].v[k] = r[i].v[k] * inv * w.v[k];
    }
  }
  if (x_out_t) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col[i] < p.width) store_pack<VEC>(x_out_t + row * p.t_pitch + col[i], r[i]);
  }
}

// ---------------------------------------------------------------------------------------------------
// xIELU over a stack of partial sums.
// ---------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
xielu_kernel(const float* __restrict__ y, int splits, int64_t split_stride, T* __restrict__ out, int n, int64_t out_pitch,
             float a, float b, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.y;
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (c >= n) return;
  const float* src = y + row * n + c;
  T* dst = out + row * out_pitch + c;
  if (vec) {
    float4 v = part_sum4(src, splits, split_stride);
    v.x = xielu_f32(v.x, a, b); v.y = xielu_f32(v.y, a, b); v.z = xielu_f32(v.z, a, b); v.w = xielu_f32(v.w, a, b);
    store4(dst, v);
  } else {
    for (int k = 0; k < 4 && c + k < n; ++k) dst[k] = from_f32<T>(xielu_f32(part_sum(src + k, splits, split_stride), a, b));
  }
}

// silu(gate) * up over a stack of partial sums [rows, 2 * padded] whose columns alternate: 16 of gate, 16 of up.
template <typename T>
__global__ void __launch_bounds__(256)
gated_silu_kernel(const float* __restrict__ y, int splits, int64_t split_stride, int64_t y_pitch, T* __restrict__ out, int n,
                  int64_t out_pitch, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.y;
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (c >= n) return;
  const float* src = y + row * y_pitch + (c >> 4) * 32 + (c & 15);
  T* dst = out + row * out_pitch + c;
  if (vec) {
    const float4 g = part_sum4(src, splits, split_stride), u = part_sum4(src + 16, splits, split_stride);
    store4(dst, make_float4(silu_f32(g.x) * u.x, silu_f32(g.y) * u.y, silu_f32(g.z) * u.z, silu_f32(g.w) * u.w));
  } else {
    for (int k = 0; k < 4 && c + k < n; ++k)
      dst[k] = from_f32<T>(silu_f32(part_sum(src + k, splits, split_stride)) * part_sum(src + 16 + k, splits, split_stride));
  }
}

// ---------------------------------------------------------------------------------------------------
// Arg-max of fp32 rows; the bits of a float are mapped to an unsigned that orders alike, then (value, index) is
// packed as in the int32 arg-max.  A NaN never wins.
// ---------------------------------------------------------------------------------------------------
__device__ __forceinline__ unsigned long long argmax_key_f32(float v, unsigned idx) {
  const unsigned u = __float_as_uint(v + 0.0f);                   // -0 becomes +0
  const unsigned ord = v != v ? 0u : ((u & 0x80000000u) ? ~u : (u | 0x80000000u));
  return ((unsigned long long)ord << 32) | (unsigned long long)(0xFFFFFFFFu - idx);
}

__global__ void __launch_bounds__(512)
argmax_f32_kernel(const float* __restrict__ logits, int64_t pitch, int64_t n, int32_t* __restrict__ out_idx) {
  __shared__ unsigned long long red[16];
  pdl_launch_dependents();
  pdl_wait();
  const float* row = logits + (int64_t)blockIdx.x * pitch;
  unsigned long long best = 0ull;
  for (int64_t c = threadIdx.x; c < n; c += 512) {
    const unsigned long long k = argmax_key_f32(row[c], (unsigned)c);
    best = k > best ? k : best;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const unsigned long long other = __shfl_xor_sync(FULL_MASK, best, o);
    best = other > best ? other : best;
  }
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = best;
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int i = 1; i < 16; ++i) best = red[i] > best ? red[i] : best;
    out_idx[blockIdx.x] = (int32_t)(0xFFFFFFFFu - (unsigned)(best & 0xFFFFFFFFull));
  }
}

template <typename T, int VEC>
static int launch_sublayer_end(const SublayerEnd& p, T* x_out_t, int64_t rows, cudaStream_t st) {
  const int groups = (p.width + VEC - 1) / VEC;
  int threads = 32;
  while (threads < 256 && threads * 2 < groups) threads *= 2;            // two groups per thread, then more threads
  while (threads < 1024 && threads * 4 < groups) threads *= 2;
  const int nv = (groups + threads - 1) / threads;
  const dim3 grid((unsigned)rows), block(threads);
  if (nv <= 1) launch_pdl(sublayer_end_kernel<T, VEC, 1>, grid, block, 0, st, p, x_out_t);
  else if (nv <= 2) launch_pdl(sublayer_end_kernel<T, VEC, 2>, grid, block, 0, st, p, x_out_t);
  else if (nv <= 4) launch_pdl(sublayer_end_kernel<T, VEC, 4>, grid, block, 0, st, p, x_out_t);
  else if (nv <= 8) launch_pdl(sublayer_end_kernel<T, VEC, 8>, grid, block, 0, st, p, x_out_t);
  else {
    set_error("sublayer_end: width %d is above the kernel's %d", p.width, 8 * 1024 * VEC);
    return B200_E_UNSUPPORTED;
  }
  return check_launch("sublayer_end");
}

template <typename T>
static int sublayer_end_typed(const SublayerEnd& p, void* x_out_t, int64_t rows, cudaStream_t st) {
  const bool vec = p.width % 4 == 0 && p.split_stride % 4 == 0 && p.plane_stride % 4 == 0 && p.t_pitch % 4 == 0 &&
                   aligned16(p.y) && aligned16(p.x_in) && aligned16(p.norm_w) && aligned16(p.x_out) && aligned16(p.hist) &&
                   aligned16(p.hist_out) && aligned16(p.final_w) && aligned16(x_out_t) && p.split_stride2 % 4 == 0 && aligned16(p.y2) &&
                   aligned16(p.w1) && aligned16(p.w2) && aligned16(p.add);
  return vec ? launch_sublayer_end<T, 4>(p, (T*)x_out_t, rows, st) : launch_sublayer_end<T, 1>(p, (T*)x_out_t, rows, st);
}

}  // namespace b200

using namespace b200;

extern "C" int b200f_embed_bigram(const void* table, const void* bigram, const int32_t* ids, const int32_t* positions,
                                  const int32_t* seq_ids, const int32_t* seq_start, const int32_t* slots,
                                  int32_t* prev_tokens, float* out, void* out_t, int dtype, int64_t tokens, int width,
                                  int64_t vocab, int64_t buckets, int64_t mul_prev, int64_t mul_cur, int64_t out_t_pitch,
                                  b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "embed: dtype %d", dtype);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && width > 0 && vocab > 0 && (!bigram || buckets > 0) && (!out_t || out_t_pitch >= width),
               B200_E_SHAPE, "embed: tokens=%lld width=%d vocab=%lld buckets=%lld", (long long)tokens, width, (long long)vocab, (long long)buckets);
  if (tokens == 0) return B200_OK;
  B200_REQUIRE(table && ids && positions && out && (!bigram || (slots && prev_tokens)) && (!seq_start == !seq_ids), B200_E_NULL,
               "embed: null pointer");
  EmbedParams p{ids, positions, seq_ids, seq_start, slots, prev_tokens, out, width, vocab, buckets, mul_prev, mul_cur, out_t_pitch};
  if (dtype == B200F_BF16)
    launch_pdl(embed_bigram_kernel<bf16>, dim3((unsigned)tokens), dim3(128), 0, (cudaStream_t)s, (const bf16*)table, (const bf16*)bigram, (bf16*)out_t, p);
  else
    launch_pdl(embed_bigram_kernel<float>, dim3((unsigned)tokens), dim3(128), 0, (cudaStream_t)s, (const float*)table, (const float*)bigram, (float*)out_t, p);
  return check_launch("embed_bigram");
}

extern "C" int b200f_sublayer_end(const float* y, int splits, int64_t split_stride, const float* y2, int splits2,
                                  int64_t split_stride2, const float* w1, const float* w2, const float* x_in,
                                  const float* norm_w, const float* add, float* x_out, void* x_out_t, const float* hist,
                                  int planes, int64_t plane_stride, const float* coef, float* hist_out, const float* final_w,
                                  int dtype, int64_t rows, int width, int64_t t_pitch, float eps, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "sublayer_end: dtype %d", dtype);
  B200_REQUIRE(rows >= 0 && rows < (1ll << 31) && width > 0 && splits >= 1 && splits2 >= 1 && planes >= 0 && (!x_out_t || t_pitch >= width), B200_E_SHAPE,
               "sublayer_end: rows=%lld width=%d splits=%d planes=%d", (long long)rows, width, splits, planes);
  if (rows == 0) return B200_OK;
  B200_REQUIRE((x_in || y) && (!y || norm_w) && (!y2 || (y && w1 && w2)) && (x_out || x_out_t) && (!coef || planes == 0 || hist), B200_E_NULL,
               "sublayer_end: null pointer");
  SublayerEnd p{y, splits, split_stride, y2, splits2, split_stride2, w1, w2, x_in, norm_w, add, x_out, hist, planes, plane_stride, coef, hist_out,
                final_w, width, t_pitch, eps};
  return dtype == B200F_BF16 ? sublayer_end_typed<bf16>(p, x_out_t, rows, (cudaStream_t)s)
                             : sublayer_end_typed<float>(p, x_out_t, rows, (cudaStream_t)s);
}

extern "C" int b200f_gated_silu(const float* y, int splits, int64_t split_stride, int64_t y_pitch, void* out, int dtype,
                                int64_t rows, int n, int64_t out_pitch, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "gated_silu: dtype %d", dtype);
  B200_REQUIRE(rows >= 0 && n > 0 && splits >= 1 && out_pitch >= n && y_pitch >= (int64_t)((n + 15) / 16) * 32, B200_E_SHAPE,
               "gated_silu: rows=%lld n=%d splits=%d", (long long)rows, n, splits);
  if (rows == 0) return B200_OK;
  B200_REQUIRE(y && out, B200_E_NULL, "gated_silu: null pointer");
  const int vec = n % 4 == 0 && split_stride % 4 == 0 && y_pitch % 4 == 0 && out_pitch % 4 == 0 && aligned16(y) && aligned16(out);
  for (int64_t r0 = 0; r0 < rows; r0 += 65535) {
    const int64_t m = rows - r0 < 65535 ? rows - r0 : 65535;
    const dim3 grid((unsigned)((n + 1023) / 1024), (unsigned)m);
    if (dtype == B200F_BF16)
      launch_pdl(gated_silu_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)s, y + r0 * y_pitch, splits, split_stride, y_pitch, (bf16*)out + r0 * out_pitch, n, out_pitch, vec);
    else
      launch_pdl(gated_silu_kernel<float>, grid, dim3(256), 0, (cudaStream_t)s, y + r0 * y_pitch, splits, split_stride, y_pitch, (float*)out + r0 * out_pitch, n, out_pitch, vec);
  }
  return check_launch("gated_silu");
}

extern "C" int b200f_xielu(const float* y, int splits, int64_t split_stride, void* out, int dtype, int64_t rows, int n,
                           int64_t out_pitch, float act_a, float act_b, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "xielu: dtype %d", dtype);
  B200_REQUIRE(rows >= 0 && rows < 65536 && n > 0 && splits >= 1 && out_pitch >= n, B200_E_SHAPE, "xielu: rows=%lld n=%d splits=%d",
               (long long)rows, n, splits);
  if (rows == 0) return B200_OK;
  B200_REQUIRE(y && out, B200_E_NULL, "xielu: null pointer");
  const int vec = n % 4 == 0 && split_stride % 4 == 0 && out_pitch % 4 == 0 && aligned16(y) && aligned16(out);
  const dim3 grid((unsigned)((n + 1023) / 1024), (unsigned)rows);
  if (dtype == B200F_BF16)
    launch_pdl(xielu_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)s, y, splits, split_stride, (bf16*)out, n, out_pitch, act_a, act_b, vec);
  else
    launch_pdl(xielu_kernel<float>, grid, dim3(256), 0, (cudaStream_t)s, y, splits, split_stride, (float*)out, n, out_pitch, act_a, act_b, vec);
  return check_launch("xielu");
}

extern "C" int b200f_argmax(const float* logits, int64_t rows, int64_t n, int64_t pitch, int32_t* out_idx, b200_stream_t s) {
  B200_REQUIRE(rows >= 0 && rows < (1ll << 31) && n > 0 && pitch >= n && n < (1ll << 31), B200_E_SHAPE, "argmax: rows=%lld n=%lld pitch=%lld",
               (long long)rows, (long long)n, (long long)pitch);
  if (rows == 0) return B200_OK;
  B200_REQUIRE(logits && out_idx, B200_E_NULL, "argmax: null pointer");
  launch_pdl(argmax_f32_kernel, dim3((unsigned)rows), dim3(512), 0, (cudaStream_t)s, logits, pitch, n, out_idx);
  return check_launch("argmax_f32");
}
