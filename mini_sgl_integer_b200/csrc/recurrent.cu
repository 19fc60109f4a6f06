// Gated linear recurrence (minGRU) over fp32 state: S_t = (1 - z_t) S_(t-1) + z_t cand_t, the gates independent of the state.
//
// Prompts: one CTA per (sequence, 32 channels).  A lane owns a channel, a warp owns kSeg consecutive tokens of the current
// stretch of kWarps * kSeg tokens.  Every warp composes its tokens' affine maps (A, B): S -> A S + B, the warps exchange the
// pairs through shared memory, and each then replays its tokens from the state in front of them; gates are read once.
// Decode: one thread per (sequence, channel).
#include "float_common.cuh"

namespace b200 {

constexpr int kScanWarps = 16;
constexpr int kScanSeg = 8;

struct MinGruParams {
  const float* zug;
  int splits;
  int64_t split_stride;
  const float *bias_z, *bias_u;
  float* state;
  const int32_t *slots, *positions, *seq_start;
  int width;
  int64_t out_pitch;
};

// (1 - z, z * candidate) of one token.
__device__ __forceinline__ void mingru_gate(float zp, float up, float* a, float* b) {
  float z;
  sigmoid_pair(zp, &z, a);
  const float cand = up >= 0.0f ? up + 0.5f : sigmoid_f32(up);
  *b = z * cand;
}

template <typename T>
__global__ void __launch_bounds__(kScanWarps * 32)
mingru_scan_kernel(const MinGruParams p, T* __restrict__ out) {
  __shared__ float2 maps[2][kScanWarps][32];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int seq = blockIdx.y, c = blockIdx.x * 32 + lane;
  const bool live = c < p.width;
  const int t0 = p.seq_start[seq], t1 = p.seq_start[seq + 1];
  if (t0 >= t1) return;
  const int64_t pitch = 3 * (int64_t)p.width;
  float* st = p.state + (int64_t)p.slots[seq] * p.width + c;
  float carry = (live && p.positions[t0] > 0) ? *st : 0.0f;
  const float bz = live ? p.bias_z[c] : 0.0f, bu = live ? p.bias_u[c] : 0.0f;
  int buf = 0;
  for (int base = t0; base < t1; base += kScanWarps * kScanSeg, buf ^= 1) {
    const int tw = base + warp * kScanSeg;
    float a[kScanSeg], b[kScanSeg], g[kScanSeg];
#pragma unroll
    for (int i = 0; i < kScanSeg; ++i) {
      a[i] = 0.0f; b[i] = 0.0f; g[i] = 0.0f;
      if (live && tw + i < t1) {
        const float* src = p.zug + (tw + i) * pitch + c;
        a[i] = part_sum(src, p.splits, p.split_stride);
        b[i] = part_sum(src + p.width, p.splits, p.split_stride);
        g[i] = part_sum(src + 2 * p.width, p.splits, p.split_stride);
      }
    }
    float A = 1.0f, B = 0.0f;
#pragma unroll
    for (int i = 0; i < kScanSeg; ++i) {
      if (tw + i < t1) {
        float ai, bi;
        mingru_gate(a[i] + bz, b[i] + bu, &ai, &bi);
        a[i] = ai; b[i] = bi;
      } else {
        a[i] = 1.0f; b[i] = 0.0f;
      }
      A *= a[i];
      B = fmaf(a[i], B, b[i]);
    }
    maps[buf][warp][lane] = make_float2(A, B);
    __syncthreads();
    float s = carry;
#pragma unroll
    for (int w = 0; w < kScanWarps; ++w) {
      if (w == warp) s = carry;
      const float2 m = maps[buf][w][lane];
      carry = fmaf(m.x, carry, m.y);
    }
#pragma unroll
    for (int i = 0; i < kScanSeg; ++i) {
      s = fmaf(a[i], s, b[i]);
      if (live && tw + i < t1) out[(int64_t)(tw + i) * p.out_pitch + c] = from_f32<T>(s * silu_f32(g[i]));
    }
  }
  if (warp == 0 && live) *st = carry;
}

template <typename T>
__global__ void __launch_bounds__(256)
mingru_step_kernel(const MinGruParams p, T* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * 256 + threadIdx.x, seq = blockIdx.y;
  if (c >= p.width) return;
  const float* src = p.zug + (int64_t)seq * 3 * p.width + c;
  float* st = p.state + (int64_t)p.slots[seq] * p.width + c;
  const float zp = part_sum(src, p.splits, p.split_stride) + p.bias_z[c];
  const float up = part_sum(src + p.width, p.splits, p.split_stride) + p.bias_u[c];
  const float g = part_sum(src + 2 * p.width, p.splits, p.split_stride);
  float s = p.positions[seq] > 0 ? *st : 0.0f;
  float a, b;
  mingru_gate(zp, up, &a, &b);
  s = fmaf(a, s, b);
  *st = s;
  out[(int64_t)seq * p.out_pitch + c] = from_f32<T>(s * silu_f32(g));
}

template <typename T>
static int mingru_typed(const MinGruParams& p, T* out, int64_t tokens, int batch, cudaStream_t st) {
  if (p.seq_start)
    launch_pdl(mingru_scan_kernel<T>, dim3((unsigned)((p.width + 31) / 32), (unsigned)batch), dim3(kScanWarps * 32), 0, st, p, out);
  else
    launch_pdl(mingru_step_kernel<T>, dim3((unsigned)((p.width + 255) / 256), (unsigned)batch), dim3(256), 0, st, p, out);
  return check_launch("mingru");
}

}  // namespace b200

using namespace b200;

extern "C" int b200f_mingru(const float* zug, int splits, int64_t split_stride, const float* bias_z, const float* bias_u,
                            float* state, const int32_t* slots, const int32_t* positions, const int32_t* seq_start,
                            void* out, int dtype, int64_t tokens, int batch, int width, int64_t out_pitch, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype), B200_E_UNSUPPORTED, "mingru: dtype %d", dtype);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && batch >= 0 && batch < 65536 && width > 0 && splits >= 1 && out_pitch >= width &&
                   (seq_start || tokens == batch),
               B200_E_SHAPE, "mingru: tokens=%lld batch=%d width=%d splits=%d", (long long)tokens, batch, width, splits);
  if (tokens == 0 || batch == 0) return B200_OK;
  B200_REQUIRE(zug && bias_z && bias_u && state && slots && positions && out, B200_E_NULL, "mingru: null pointer");
  MinGruParams p{zug, splits, split_stride, bias_z, bias_u, state, slots, positions, seq_start, width, out_pitch};
  return dtype == B200F_BF16 ? mingru_typed<bf16>(p, (bf16*)out, tokens, batch, (cudaStream_t)s)
                             : mingru_typed<float>(p, (float*)out, tokens, batch, (cudaStream_t)s);
}
