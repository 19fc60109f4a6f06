// Matrix-valued recurrences: per head a state S [dim, vdim] in 32-bit,
//
//   S_t = a_t S_(t-1) + k_t w_t^T,      o_t = S_t^T q_t        (S of the current token: the read-out sees its own write)
//
//   B200F_MEMORY_EXP    a = exp(f + m_(t-1) - m_t), w = exp(i - m_t) v with the running maximum m_t = max(f + m_(t-1), i),
//                       m_0 = 0; a vector n follows the same recurrence with w = 1 scale, and the read-out is divided by
//                       max(|n . q|, exp(-m_t)) + 1e-6
//   B200F_MEMORY_SSD    a = exp(-exp(A_log) dt), w = dt v, plus a skip D v on the read-out
//   B200F_MEMORY_DELTA  q and k made unit vectors, w = beta (v - a S_(t-1)^T k)
//
// memory_prepare_kernel   between the projections and the recurrence: the optional short causal convolution with silu, the
//                         split into heads (each padded to 8 values), and the gates.  A token block per CTA, a channel (or
//                         four) per thread with the taps in registers.  conv_state_kernel leaves the last inputs for the
//                         sequence's next portion.
// memory_chunk_kernel     prompts in bf16, 64 tokens at a time on the tensor cores, see below.
// memory_scan_kernel      prompts, any type and size (the 32-bit path; short portions): a CTA per (sequence, head, slice of columns) keeps its part of S in registers over all
//                         tokens: LN lanes share a column quad, each holds R of its rows as fp32 pairs.  Tokens come
//                         through shared memory in stages of 16.  Tokens are processed one by one in the order of the
//                         equations, so how a prompt was cut makes no difference at all.
// memory_step_kernel      decode: streams S through registers once.
// memory_output_kernel    read-out -> (gate,) norm per group (, gate) -> operand of the output projection.
#include "float_common.cuh"
#include "umma.cuh"

namespace b200 {

constexpr float kUnitEps = 1e-6f;      // under the root of a unit vector, and added to the normaliser of the read-out

// ---------------------------------------------------------------------------------------------------
struct MemoryPrepare {
  const float* y;
  int splits;
  int64_t split_stride, y_pitch, col0;
  int channels;
  const float *conv_w, *conv_b;
  int taps;                            // 0: no convolution and no activation
  float* conv_state;                   // [slots][taps - 1][channels]
  const int32_t *slots, *positions, *seq_start, *seq_ids;
  int seg_width[3], seg_head[3];       // the channels are three segments of heads
  int64_t out_pitch;
  int kind, heads;
  int64_t gate_col_a, gate_col_b;
  const float *gate_a, *gate_b;
  float cap;
  float4* gates;                       // [tokens][heads]
  float* norm_state;                   // EXP: [slots][heads][dim + 1], the last entry is the maximum
  int norm_dim;
  int64_t tokens;
  int block_tokens, channel_blocks;
};

__device__ __forceinline__ int pad8i(int n) { return (n + 7) & ~7; }

// Column of channel c in a row of padded heads.
__device__ __forceinline__ int padded_column(const MemoryPrepare& p, int c) {
  int out = 0;
#pragma unroll
  for (int s = 0; s < 3; ++s) {
    const int w = p.seg_width[s], h = p.seg_head[s];
    if (c < w) return h == 0 ? out + c : out + (c / h) * pad8i(h) + c % h;
    c -= w;
    if (h) out += (w / h) * pad8i(h);
  }
  return out;
}

// (first, second) gate of one token and head: EXP log gates (f, i), SSD (log decay, dt), DELTA (log decay, beta).
__device__ __forceinline__ float2 memory_gates(const MemoryPrepare& p, const float* row, int h) {
  const float a = part_sum(row + p.gate_col_a + h, p.splits, p.split_stride);
  if (p.kind == B200F_MEMORY_EXP) {
    const float b = part_sum(row + p.gate_col_b + h, p.splits, p.split_stride);
    const float f = p.cap * tanhf((a + p.gate_a[h]) / p.cap), i = p.cap * tanhf((b + p.gate_b[h]) / p.cap);
    return make_float2(-softplus_f32(-f), i);
  }
  const float dt = softplus_f32(a + p.gate_b[h]);
  const float log_decay = -expf(p.gate_a[h]) * dt;
  if (p.kind == B200F_MEMORY_SSD) return make_float2(log_decay, dt);
  return make_float2(log_decay, sigmoid_f32(part_sum(row + p.gate_col_b + h, p.splits, p.split_stride)));
}

template <typename T, int VEC, int TAPS>      // TAPS 0: none, -1: any number
__global__ void __launch_bounds__(256)
memory_prepare_kernel(const MemoryPrepare p, T* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t t_lo = (int64_t)blockIdx.y * p.block_tokens, t_hi = min(t_lo + p.block_tokens, p.tokens);
  if ((int)blockIdx.x >= p.channel_blocks) {
    const int n = (int)(t_hi - t_lo) * p.heads;
    for (int i = (blockIdx.x - p.channel_blocks) * 256 + threadIdx.x; i < n; i += (gridDim.x - p.channel_blocks) * 256) {
      const int64_t t = t_lo + i / p.heads;
      const int h = i % p.heads;
      const float2 g = memory_gates(p, p.y + t * p.y_pitch, h);
      float4 r = make_float4(g.x, g.y, 0.0f, 0.0f);
      if (p.kind == B200F_MEMORY_EXP && !p.seq_start) {           // decode: this thread moves the maximum on
        float* ms = p.norm_state + ((int64_t)p.slots[t] * p.heads + h) * (p.norm_dim + 1) + p.norm_dim;
        const float m0 = p.positions[t] > 0 ? *ms : 0.0f, fm = g.x + m0, m = fmaxf(fm, g.y);
        *ms = m;
        r = make_float4(fm - m, expf(g.y - m), expf(-m), 0.0f);
      }
      p.gates[t * p.heads + h] = r;
    }
    return;
  }
  const int c = (blockIdx.x * 256 + threadIdx.x) * VEC;
  if (c >= p.channels) return;
  const int oc = padded_column(p, c);
  const float* col = p.y + p.col0 + c;
  auto load = [&](int64_t t, float (&v)[VEC]) {
    if (VEC == 4) {
      const float4 f = part_sum4(col + t * p.y_pitch, p.splits, p.split_stride);
      v[0] = f.x; v[VEC > 1 ? 1 : 0] = f.y; v[VEC > 2 ? 2 : 0] = f.z; v[VEC > 3 ? 3 : 0] = f.w;
    } else {
      v[0] = part_sum(col + t * p.y_pitch, p.splits, p.split_stride);
    }
  };
  auto store = [&](int64_t t, const float (&v)[VEC]) {
    T* dst = out + t * p.out_pitch + oc;
    if (VEC == 4) store4(dst, make_float4(v[0], v[VEC > 1 ? 1 : 0], v[VEC > 2 ? 2 : 0], v[VEC > 3 ? 3 : 0]));
    else dst[0] = from_f32<T>(v[0]);
  };
  if (TAPS == 0) {
    for (int64_t t = t_lo; t < t_hi; ++t) {
      float v[VEC];
      load(t, v);
      store(t, v);
    }
    return;
  }
  const int taps = TAPS > 0 ? TAPS : p.taps;
  // input at `back` tokens in front of token t of sequence seq, whose first new token is `first`
  auto input = [&](int64_t t, int64_t first, int slot, int pos, int back, float (&v)[VEC]) {
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = 0.0f;
    if (pos < back) return;
    const int64_t local = t - first - back;
    if (local >= 0) {
      load(t - back, v);
    } else {
      const float* s = p.conv_state + ((int64_t)slot * (taps - 1) + (taps - 1) + local) * p.channels + c;
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[k] = s[k];
    }
  };
  constexpr int H = TAPS > 0 ? TAPS : 1;
  float hist[H][VEC], w[H][VEC], bias[VEC];
#pragma unroll
  for (int k = 0; k < VEC; ++k) bias[k] = p.conv_b ? p.conv_b[c + k] : 0.0f;
  if (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < H; ++j)
#pragma unroll
      for (int k = 0; k < VEC; ++k) w[j][k] = p.conv_w[(int64_t)(c + k) * taps + j];
  }
  int seq = -1;
  for (int64_t t = t_lo; t < t_hi; ++t) {
    const int s = p.seq_start ? p.seq_ids[t] : (int)t;
    const int64_t first = p.seq_start ? p.seq_start[s] : t;
    const int slot = p.slots[s], pos = p.positions[t];
    float acc[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) acc[k] = bias[k];
    if (TAPS > 0) {
      if (s != seq) {
#pragma unroll
        for (int j = 1; j < H; ++j) input(t, first, slot, pos, H - j, hist[j]);    // moved down by one below
      }
#pragma unroll
      for (int j = 0; j + 1 < H; ++j)
#pragma unroll
        for (int k = 0; k < VEC; ++k) hist[j][k] = hist[j + 1][k];
      load(t, hist[H - 1]);
#pragma unroll
      for (int j = 0; j < H; ++j)
#pragma unroll
        for (int k = 0; k < VEC; ++k) acc[k] = fmaf(w[j][k], hist[j][k], acc[k]);
      if (!p.seq_start) {
        float* st = p.conv_state + (int64_t)slot * (H - 1) * p.channels + c;
#pragma unroll
        for (int j = 1; j < H; ++j)
#pragma unroll
          for (int k = 0; k < VEC; ++k) st[(int64_t)(j - 1) * p.channels + k] = hist[j][k];
      }
    } else {
      for (int j = 0; j < taps; ++j) {
        float v[VEC];
        input(t, first, slot, pos, taps - 1 - j, v);
#pragma unroll
        for (int k = 0; k < VEC; ++k) acc[k] = fmaf(p.conv_w[(int64_t)(c + k) * taps + j], v[k], acc[k]);
      }
      if (!p.seq_start && taps > 1) {
        float* st = p.conv_state + (int64_t)slot * (taps - 1) * p.channels + c;
        float v[VEC];
        load(t, v);
        for (int j = 0; j < taps - 1; ++j)
#pragma unroll
          for (int k = 0; k < VEC; ++k) st[(int64_t)j * p.channels + k] = j + 1 < taps - 1 ? st[(int64_t)(j + 1) * p.channels + k] : v[k];
      }
    }
    seq = s;
#pragma unroll
    for (int k = 0; k < VEC; ++k) acc[k] = silu_f32(acc[k]);
    store(t, acc);
  }
}

// The last taps - 1 inputs of every sequence of a prompt batch; runs after memory_prepare_kernel has read the old ones.
__global__ void __launch_bounds__(256)
conv_state_kernel(const MemoryPrepare p) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * 256 + threadIdx.x, seq = blockIdx.y;
  if (c >= p.channels) return;
  const int64_t first = p.seq_start[seq], count = p.seq_start[seq + 1] - first;
  if (count <= 0) return;
  const int keep = p.taps - 1;
  float* st = p.conv_state + (int64_t)p.slots[seq] * keep * p.channels + c;
  for (int i = 0; i < keep; ++i) {                                  // reads entry i + count, writes entry i
    const int64_t local = count - keep + i;
    st[(int64_t)i * p.channels] = local >= 0 ? part_sum(p.y + (first + local) * p.y_pitch + p.col0 + c, p.splits, p.split_stride)
                                             : st[(keep + local) * p.channels];
  }
}

// ---------------------------------------------------------------------------------------------------
struct MemoryParams {
  int64_t row_pitch;
  int64_t q_off, k_off, v_off;         // columns in a row; heads are padded to 8 values
  int qk_heads, heads, dim, vdim;
  float4* gates;
  float q_scale;
  const float* skip;                   // nullable, [heads]
  float* state;                        // [slots][heads][dim][pad8(vdim)]
  float* norm_state;                   // EXP: [slots][heads][dim + 1]
  const int32_t *slots, *positions, *seq_start;
  float* out;                          // [tokens][heads * vdim]
  float* den;                          // EXP: [tokens][heads]
  int warps;
};

constexpr int kStageTokens = 16;

// Four column sums spread over LN lanes: afterwards every lane has the total of column reduced_column(lane).
template <int LN>
__device__ __forceinline__ float reduce4(const float (&v)[4], int ln) {
  const bool b0 = ln & 1, b1 = ln & 2;
  float k0 = b0 ? v[2] : v[0], k1 = b0 ? v[3] : v[1];
  k0 += __shfl_xor_sync(FULL_MASK, b0 ? v[0] : v[2], 1);
  k1 += __shfl_xor_sync(FULL_MASK, b0 ? v[1] : v[3], 1);
  float k = b1 ? k1 : k0;
  k += __shfl_xor_sync(FULL_MASK, b1 ? k0 : k1, 2);
#pragma unroll
  for (int o = 4; o < LN; o <<= 1) k += __shfl_xor_sync(FULL_MASK, k, o);
  return k;
}
__device__ __forceinline__ int reduced_column(int ln) { return (ln & 1) * 2 + ((ln >> 1) & 1); }

template <typename T>
struct ScanShape {
  int np, vs, vsp, hq;
  __host__ __device__ ScanShape(int np_, int dim, int vs_) : np(np_), vs(vs_), vsp((vs_ + 7) & ~7), hq((dim + 7) & ~7) {}
  __host__ __device__ int raw_row() const { return 2 * hq + vsp; }                              // values of T
  __host__ __device__ size_t raw_bytes() const { return ((size_t)kStageTokens * raw_row() * sizeof(T) + kStageTokens * 16 + 15) & ~size_t(15); }
  __host__ __device__ size_t bytes() const { return 2 * raw_bytes() + (size_t)kStageTokens * (2 * np + vsp + 4) * 4; }
};

template <typename T, int KIND, int LN, int R>
__global__ void __launch_bounds__(288)
memory_scan_kernel(const MemoryParams p, const T* __restrict__ rows) {
  extern __shared__ __align__(16) unsigned char smem[];
  constexpr int NP = LN * R, CPW = (32 / LN) * 4, TB = kStageTokens;
  const int W = p.warps, VS = CPW * W;
  const ScanShape<T> sh(NP, p.dim, VS);
  const int hq = sh.hq, vsp = sh.vsp, raw_row = sh.raw_row();
  unsigned char* raw0 = smem;
  float* qf = reinterpret_cast<float*>(smem + 2 * sh.raw_bytes());
  float* kf = qf + TB * NP;
  float* vf = kf + TB * NP;
  float* sc = vf + TB * vsp;

  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, threads = blockDim.x, nwarps = threads >> 5;
  const int slice = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int64_t t0 = p.seq_start[seq];
  const int count = p.seq_start[seq + 1] - (int)t0;
  if (count <= 0) return;
  const int vp = pad8i(p.vdim), col0 = slice * VS;
  const int qh = h / (p.heads / p.qk_heads);
  const T* q_src = rows + p.q_off + (int64_t)qh * hq;
  const T* k_src = rows + p.k_off + (int64_t)qh * hq;
  const T* v_src = rows + p.v_off + (int64_t)h * vp + col0;
  const bool has_state = p.positions[t0] > 0;
  const int64_t slot_head = (int64_t)p.slots[seq] * p.heads + h;

  constexpr int PER = 16 / sizeof(T);                 // values per copied chunk
  const int cq = hq / PER, cv = vsp / PER, chunks = 2 * cq + cv + 1;
  auto issue = [&](int stage) {
    const int base = stage * TB, n = min(TB, count - base);
    unsigned char* raw = raw0 + (stage & 1) * sh.raw_bytes();
    for (int i = tid; i < n * chunks; i += threads) {
      const int t = i / chunks, c = i - t * chunks;
      const int64_t tok = t0 + base + t;
      T* dst = reinterpret_cast<T*>(raw) + t * raw_row;
      if (c < cq) cp_async16(smem_u32(dst + c * PER), q_src + tok * p.row_pitch + c * PER);
      else if (c < 2 * cq) cp_async16(smem_u32(dst + c * PER), k_src + tok * p.row_pitch + (c - cq) * PER);
      else if (c < 2 * cq + cv) {
        const int vc = (c - 2 * cq) * PER;
        if (col0 + vc < vp) cp_async16(smem_u32(dst + 2 * hq + vc), v_src + tok * p.row_pitch + vc);
      } else {
        cp_async16(smem_u32(raw + sh.raw_bytes() - TB * 16 + t * 16), p.gates + tok * p.heads + h);
      }
    }
    cp_async_commit();
  };

  const int ln = lane % LN, cg = lane / LN;
  const int c_local = warp * CPW + cg * 4, c_glob = col0 + c_local;
  const bool consumer = warp < W;
  f32x2 S[R / 2][4];
#pragma unroll
  for (int r = 0; r < R / 2; ++r)
#pragma unroll
    for (int c = 0; c < 4; ++c) S[r][c] = 0ull;
  float* st = p.state + slot_head * p.dim * vp + c_glob;
  if (consumer && has_state && c_glob < vp) {
#pragma unroll
    for (int r = 0; r < R; r += 2) {
      const int n = ((r / 4) * LN + ln) * 4 + (r & 2);
      const float4 z = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      const float4 a = n < p.dim ? *reinterpret_cast<const float4*>(st + (int64_t)n * vp) : z;
      const float4 b = n + 1 < p.dim ? *reinterpret_cast<const float4*>(st + (int64_t)(n + 1) * vp) : z;
      S[r / 2][0] = pack2(a.x, b.x); S[r / 2][1] = pack2(a.y, b.y); S[r / 2][2] = pack2(a.z, b.z); S[r / 2][3] = pack2(a.w, b.w);
    }
  }
  // the extra warp of the EXP kind runs the normaliser, in the first slice's CTA
  constexpr int NV = (NP + 31) / 32;
  float nv[NV];
  float* nst = KIND == B200F_MEMORY_EXP ? p.norm_state + slot_head * (p.dim + 1) : nullptr;
  const bool normaliser = KIND == B200F_MEMORY_EXP && warp == W && slice == 0;
  if (normaliser) {
#pragma unroll
    for (int i = 0; i < NV; ++i) nv[i] = (has_state && lane + 32 * i < p.dim) ? nst[lane + 32 * i] : 0.0f;
  }
  const float skip = p.skip ? p.skip[h] : 0.0f;
  const int my_col = c_glob + reduced_column(ln);
  float* out = p.out + t0 * p.heads * p.vdim + (int64_t)h * p.vdim + my_col;
  const bool writes = consumer && ln < 4 && my_col < p.vdim;

  const int stages = (count + TB - 1) / TB;
  issue(0);
  for (int s = 0; s < stages; ++s) {
    const int n = min(TB, count - s * TB);
    cp_async_wait<0>();
    __syncthreads();                                  // stage s is here; everyone is done with stage s - 1
    if (s + 1 < stages) issue(s + 1);
    const unsigned char* raw = raw0 + (s & 1) * sh.raw_bytes();
    const float4* rg = reinterpret_cast<const float4*>(raw + sh.raw_bytes() - TB * 16);
    for (int t = warp; t < n; t += nwarps) {
      const T* src = reinterpret_cast<const T*>(raw) + t * raw_row;
      float sq = 0.0f, sk = 0.0f;
      for (int i = lane; i < NP; i += 32) {
        const float q = i < p.dim ? to_f32(src[i]) : 0.0f, k = i < p.dim ? to_f32(src[hq + i]) : 0.0f;
        qf[t * NP + i] = q;
        kf[t * NP + i] = k;
        sq = fmaf(q, q, sq);
        sk = fmaf(k, k, sk);
      }
      for (int i = lane; i < vsp; i += 32) vf[t * vsp + i] = col0 + i < p.vdim ? to_f32(src[2 * hq + i]) : 0.0f;
      if (KIND == B200F_MEMORY_DELTA) {
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if (lane == 0) *reinterpret_cast<float4*>(sc + 4 * t) = make_float4(expf(rg[t].x), rg[t].y, 1.0f / sqrtf(sk + kUnitEps), p.q_scale / sqrtf(sq + kUnitEps));
      } else if (lane == 0) {
        *reinterpret_cast<float4*>(sc + 4 * t) = make_float4(expf(rg[t].x), rg[t].y, rg[t].z, p.q_scale);
      }
    }
    __syncthreads();
    if (consumer) {
#pragma unroll 1
      for (int t = 0; t < n; ++t) {
        const float4 g = *reinterpret_cast<const float4*>(sc + 4 * t);      // decay, write strength, 1 / |k| or exp(-m), scale of q
        const float4 v4 = *reinterpret_cast<const float4*>(vf + t * vsp + c_local);
        f32x2 k2[R / 2], q2[R / 2];
#pragma unroll
        for (int r = 0; r < R / 4; ++r) {
          const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(kf + t * NP + (r * LN + ln) * 4);
          const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(qf + t * NP + (r * LN + ln) * 4);
          k2[2 * r] = kk.x; k2[2 * r + 1] = kk.y;
          q2[2 * r] = qq.x; q2[2 * r + 1] = qq.y;
        }
        float w[4] = {g.y * v4.x, g.y * v4.y, g.y * v4.z, g.y * v4.w};
        if (KIND == B200F_MEMORY_DELTA) {
          f32x2 d2[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
          for (int r = 0; r < R / 2; ++r)
#pragma unroll
            for (int c = 0; c < 4; ++c) d2[c] = fma2(S[r][c], k2[r], d2[c]);
          float d[4];
#pragma unroll
          for (int c = 0; c < 4; ++c) { const float2 u = unpack2(d2[c]); d[c] = u.x + u.y; }
          const float mine = reduce4<LN>(d, ln);
          const int src = lane & ~(LN - 1);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float dc = __shfl_sync(FULL_MASK, mine, src | (c >> 1) | ((c & 1) << 1));
            w[c] = (w[c] - g.y * g.x * g.z * dc) * g.z;
          }
        }
        const f32x2 aa = pack2(g.x, g.x);
        f32x2 o2[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const f32x2 ww = pack2(w[c], w[c]);
#pragma unroll
          for (int r = 0; r < R / 2; ++r) {
            S[r][c] = fma2(k2[r], ww, mul2(S[r][c], aa));
            o2[c] = fma2(S[r][c], q2[r], o2[c]);
          }
        }
        float o[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) { const float2 u = unpack2(o2[c]); o[c] = u.x + u.y; }
        float mine = reduce4<LN>(o, ln) * g.w;
        if (KIND == B200F_MEMORY_SSD) mine = fmaf(skip, vf[t * vsp + c_local + reduced_column(ln)], mine);
        if (writes) out[(int64_t)(s * TB + t) * p.heads * p.vdim] = mine;
      }
    } else if (normaliser) {
      for (int t = 0; t < n; ++t) {
        const float4 g = *reinterpret_cast<const float4*>(sc + 4 * t);
        float dot = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int e = lane + 32 * i;
          const float k = e < NP ? kf[t * NP + e] : 0.0f, q = e < NP ? qf[t * NP + e] : 0.0f;
          nv[i] = fmaf(g.y, k, g.x * nv[i]);
          dot = fmaf(nv[i], q, dot);
        }
        dot = warp_sum(dot) * p.q_scale;
        if (lane == 0) p.den[(t0 + s * TB + t) * p.heads + h] = fmaxf(fabsf(dot), g.z) + kUnitEps;
      }
    }
  }
  if (consumer && c_glob < vp) {
#pragma unroll
    for (int r = 0; r < R; r += 2) {
      const int n = ((r / 4) * LN + ln) * 4 + (r & 2);
      const float2 a = unpack2(S[r / 2][0]), b = unpack2(S[r / 2][1]), c = unpack2(S[r / 2][2]), d = unpack2(S[r / 2][3]);
      if (n < p.dim) *reinterpret_cast<float4*>(st + (int64_t)n * vp) = make_float4(a.x, b.x, c.x, d.x);
      if (n + 1 < p.dim) *reinterpret_cast<float4*>(st + (int64_t)(n + 1) * vp) = make_float4(a.y, b.y, c.y, d.y);
    }
  }
  if (normaliser) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (lane + 32 * i < p.dim) nst[lane + 32 * i] = nv[i];
  }
}

// Log gates (f, i) of a prompt batch to (f + m_(t-1) - m_t, exp(i - m_t), exp(-m_t)); a warp per (sequence, head).
__global__ void __launch_bounds__(32)
running_max_kernel(const MemoryPrepare p) {
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, seq = blockIdx.y, lane = threadIdx.x;
  const int64_t t0 = p.seq_start[seq], t1 = p.seq_start[seq + 1];
  if (t0 >= t1) return;
  float* ms = p.norm_state + ((int64_t)p.slots[seq] * p.heads + h) * (p.norm_dim + 1) + p.norm_dim;
  float m = p.positions[t0] > 0 ? *ms : 0.0f;
  const float4 none = make_float4(0.0f, -INFINITY, 0.0f, 0.0f);         // leaves the maximum alone
  auto load = [&](int64_t t) { return t < t1 ? p.gates[t * p.heads + h] : none; };
  float4 next[2] = {load(t0 + lane), load(t0 + 32 + lane)};
  for (int64_t base = t0; base < t1; base += 32) {
    const float4 g = next[0];
    next[0] = next[1];
    next[1] = load(base + 64 + lane);
    float a = g.x, b = g.y;                              // m -> max(m + a, b), composed over the lanes up to this one
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pa = __shfl_up_sync(FULL_MASK, a, o), pb = __shfl_up_sync(FULL_MASK, b, o);
      if (lane >= o) {
        b = fmaxf(pb + a, b);
        a += pa;
      }
    }
    const float after = fmaxf(m + a, b);
    float before = __shfl_up_sync(FULL_MASK, after, 1);
    if (lane == 0) before = m;
    m = __shfl_sync(FULL_MASK, after, 31);
    if (base + lane < t1) p.gates[(base + lane) * p.heads + h] = make_float4(fminf(g.x + before - after, 0.0f), expf(g.y - after), expf(-after), 0.0f);
  }
  if (lane == 0) *ms = m;
}

// ---------------------------------------------------------------------------------------------------
// Chunks of 64 tokens.  With L_t the sum of the chunk's log decays up to token t, and S_0 the state in front of it,
//
//   o_t = e^(L_t) S_0^T q_t + sum_(s <= t) (q_t . k_s) e^(L_t - L_s) w_s          w_s: the written vector without the decay
//   S   = e^(L_64) S_0 + sum_s k_s (e^(L_64 - L_s) w_s)^T
//
// Every exponent is <= 0.  EXP and SSD know w_s = b_s v_s.  For DELTA the written vectors U solve
// (I + M) U = diag(beta) (V - diag(e^L) K S_0), M_ts = beta_t e^(L_t - L_s) (k_t . k_s) for s < t; delta_inverse_kernel
// computes (I + M)^-1 for all chunks at once, so that only matrix products are left on the way from chunk to chunk.
//
// q, k and v are bf16.  S lives in fp32 accumulators; where S, decayed scores, U or the inverse are operands of a product,
// they are the sum of two bf16 numbers (16 bits of fraction) and the small terms' product is left out.
//
// A CTA per (sequence, head, 64 columns); each of 4 warps owns 16 columns and holds S^T [16, dim] in accumulators over all
// chunks.  With everything transposed, an accumulator tile has the layout of the left operand of the next product, so S, the
// right-hand side and U never leave the registers; shared memory holds q, k, v, the decayed scores and the inverse, each
// read as the right operand.  EXP: the CTA of the first columns also runs the normaliser, n . q = e^L (n_0 . q) + the row sums
// of the decayed scores, on the fp32 units.
// ---------------------------------------------------------------------------------------------------
constexpr int kChunk = 64, kChunkWarps = 4, kChunkCols = 16 * kChunkWarps;
constexpr int kPanel = kChunk * 128;     // bytes of 64 rows of 64 bf16 values, as TMA writes them with the 128-byte swizzle


__device__ __forceinline__ void mm_ldsm(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mm_ldsm_t(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mm_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float exp2_fast(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}
// (a, b) as the sum of two pairs of bf16.
__device__ __forceinline__ void split2(float a, float b, unsigned* hi, unsigned* lo) {
  *hi = f32_to_bf16x2(a, b);
  const float2 h = bf16x2_to_f32(*hi);
  *lo = f32_to_bf16x2(a - h.x, b - h.y);
}
__device__ __forceinline__ void cp_async16_or_zero(unsigned dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}

__device__ __forceinline__ void bulk_copy(unsigned dst, const void* src, unsigned bytes, unsigned bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// Orders this thread's accesses to shared memory in front of later bulk copies into it (behind a barrier).
__device__ __forceinline__ void async_fence() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

// Where a sequence's chunks lie among those of the batch.
__device__ __forceinline__ int64_t chunk_index(int64_t first_token, int seq, int chunk) { return first_token / kChunk + seq + chunk; }

__host__ __device__ constexpr int chunk_panels(int dr) { return dr <= 4 ? 1 : dr / 4; }
__host__ __device__ constexpr size_t chunk_smem(int dr, int kind) {
  return (size_t)(2 * (2 * chunk_panels(dr) + 1) + (kind == B200F_MEMORY_DELTA ? 3 : 2)) * kPanel + 12 * kChunk * 4 + 2 * kChunk * 16 +
         (kind == B200F_MEMORY_EXP ? (9 * 16 * dr + 4 * kChunk) * 4 : 0) + 24 + 1024;
}
// Byte offset of (row, col) in a panel.
__host__ __device__ __forceinline__ int panel_at(int row, int col) { return row * 128 + ((((col >> 3) ^ row) & 7) << 4) + (col & 7) * 2; }

// Inclusive sums of 64 values, two per lane (token = lane, lane + 32), by one warp.
__device__ __forceinline__ void sum64(float& a, float& b, int lane) {
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float x = __shfl_up_sync(FULL_MASK, a, o), y = __shfl_up_sync(FULL_MASK, b, o);
    if (lane >= o) { a += x; b += y; }
  }
  b += __shfl_sync(FULL_MASK, a, 31);
}

template <int KIND, int DR, bool FULL>      // FULL: dim is exactly 16 DR
__global__ void __launch_bounds__(kChunkWarps * 32, DR > 8 ? 1 : 2)
memory_chunk_kernel(const __grid_constant__ CUtensorMap map, const MemoryParams p, const bf16* __restrict__ inverse) {
  extern __shared__ __align__(16) unsigned char smem[];
  constexpr bool DELTA = KIND == B200F_MEMORY_DELTA, EXP = KIND == B200F_MEMORY_EXP;
  constexpr int C = kChunk, THREADS = kChunkWarps * 32, DP = chunk_panels(DR);
  // panels: twice (q [DP], k [DP], v), for this chunk and the next, then the decayed scores' low and high parts (DELTA: the high
  // part takes the place of v, which is used up by then) and, DELTA, the inverse's high and low parts
  constexpr int K_ = DP, V_ = 2 * DP, NB = 2 * DP + 1, PL_ = 2 * NB, PH_ = DELTA ? V_ : PL_ + 1, T_ = PL_ + 1;
  const unsigned p_base = (smem_u32(smem) + 1023) & ~1023u;
  unsigned char* panels = smem + (p_base - smem_u32(smem));
  // per token, for this chunk and the next: L in units of log2; e^L; write strength; exp(-m) or 1 / |k|; scale of q; e^(L_64 - L)
  // times the strength or 1 / |k|
  float* token_values = reinterpret_cast<float*>(panels + (PL_ + (DELTA ? 3 : 2)) * kPanel);

  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, q2 = 2 * (lane & 3);
  const int slice = blockIdx.x, h = blockIdx.y, seq = blockIdx.z, col0 = slice * kChunkCols;
  const int vp = p.vdim, k16 = p.dim >> 4, qh = h / (p.heads / p.qk_heads);
  float4* gs = reinterpret_cast<float4*>(token_values + 12 * C);        // [2][C]
  float *ns = reinterpret_cast<float*>(gs + 2 * C), *nsum = ns + (EXP ? 16 * DR : 0), *np = nsum + (EXP ? 4 * C : 0);   // EXP: n, row sums of the scores by column block, parts of n's update
  const unsigned bar = smem_u32(np + (EXP ? 8 * 16 * DR : 0));
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(bar + 8 * i, 1);                // this chunk, the next; the inverse
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  pdl_wait();
  const int64_t t0 = p.seq_start[seq];
  const int count = p.seq_start[seq + 1] - (int)t0;
  if (count <= 0) return;
  const bool has_state = p.positions[t0] > 0;
  const bool with_n = EXP && slice == 0, works = col0 + warp * 16 < vp;
  const int64_t slot_head = (int64_t)p.slots[seq] * p.heads + h;
  const int64_t q_col = p.q_off + (int64_t)qh * p.dim, k_col = p.k_off + (int64_t)qh * p.dim, v_col = p.v_off + (int64_t)h * vp + col0;

  const float skip = KIND == B200F_MEMORY_SSD && p.skip ? p.skip[h] / p.q_scale : 0.0f;

  // S^T: rows are columns col0 + 16 warp + g (+ 8) of S, accumulator columns its rows
  float S[2 * DR][4];
  const int c_lo = warp * 16 + g, c_hi = c_lo + 8;       // within the slice
  float* st = p.state + slot_head * p.dim * vp + col0;
  float* nst = EXP ? p.norm_state + slot_head * (p.dim + 1) : nullptr;
#pragma unroll
  for (int i = 0; i < 2 * DR; ++i)
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int d = i * 8 + q2 + (k & 1), c = k < 2 ? c_lo : c_hi;
      float v = 0.0f;
      if (has_state && works && (FULL || d < p.dim)) {
        if (col0 + c < vp) v = st[(int64_t)d * vp + c];
      }
      S[i][k] = v;
    }

  // ldmatrix addresses: rows of 128 bytes, 16-byte pieces exchanged by the row's last three bits
  if (with_n)
    for (int d = tid; d < 16 * DR; d += THREADS) ns[d] = has_state && d < p.dim ? nst[d] : 0.0f;
  const unsigned n_row = ((lane & 7) + ((lane >> 4) << 3)) * 128, n_x = (((lane >> 3) & 1) ^ (lane & 7)) << 4;     // right operand from [n][k], left from [k][m]
  const unsigned m_row = (lane & 15) * 128, m_x = ((lane >> 4) ^ (lane & 7)) << 4;                                 // left operand from [m][k], right from [k][n]
  unsigned n_at[4], m_at[4], n_fix[4];                   // in the current chunk's panels, and in those there are one of
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    n_fix[i] = n_at[i] = p_base + n_row + (n_x ^ (i << 5));
    m_at[i] = p_base + m_row + (m_x ^ (i << 5));
  }
  unsigned v_at = p_base + V_ * kPanel + n_row + (n_x ^ ((warp & 3) << 5));
  auto at_n = [&](int panel, int row16, int k16th) { return n_at[k16th & 3] + (panel + (k16th >> 2)) * kPanel + row16 * 2048; };
  auto at_m = [&](int panel, int row16, int k16th) { return m_at[k16th & 3] + (panel + (k16th >> 2)) * kPanel + row16 * 2048; };
  auto at_fix = [&](int panel, int row16, int k16th) { return n_fix[k16th & 3] + (panel + (k16th >> 2)) * kPanel + row16 * 2048; };

  // acc [16 columns, 64 tokens] = S^T X^T for X = q or k
  auto state_times = [&](int x, float (&acc)[8][4]) {
#pragma unroll
    for (int kk = 0; kk < DR; ++kk) {
      if (!FULL && kk >= k16) break;
      unsigned ah[4], al[4];
      split2(S[2 * kk][0], S[2 * kk][1], &ah[0], &al[0]);
      split2(S[2 * kk][2], S[2 * kk][3], &ah[1], &al[1]);
      split2(S[2 * kk + 1][0], S[2 * kk + 1][1], &ah[2], &al[2]);
      split2(S[2 * kk + 1][2], S[2 * kk + 1][3], &ah[3], &al[3]);
      unsigned b[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) mm_ldsm(b[j], at_n(x, j, kk));
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        mm_mma(acc[2 * j], ah, b[j][0], b[j][1]);
        mm_mma(acc[2 * j + 1], ah, b[j][2], b[j][3]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        mm_mma(acc[2 * j], al, b[j][0], b[j][1]);
        mm_mma(acc[2 * j + 1], al, b[j][2], b[j][3]);
      }
    }
  };
  // V^T of 16 tokens as a left operand; in the accumulator layout: pairs of tokens
  auto values = [&](int kb, unsigned (&a)[4]) { mm_ldsm_t(a, v_at + kb * 2048); };

  const int chunks = (count + C - 1) / C;
  auto load_gates = [&](int ch) {                         // by warp 0, a chunk ahead; entries behind the portion are not used
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = lane + 32 * half;
      if (ch * C + t < count) cp_async16(smem_u32(gs + (ch & 1) * C + t), p.gates + (t0 + (int64_t)ch * C + t) * p.heads + h);
    }
    cp_async_commit();
  };
  auto load_chunk = [&](int ch) {                         // by the first lane of every warp: an issue takes long, so they share
    const unsigned to = p_base + (ch & 1) * NB * kPanel, b = bar + 8 * (ch & 1);
    const int tok = (int)(t0 + (int64_t)ch * C);
    if (warp == 1) {
      mbar_expect_tx(b, NB * kPanel);
      tma_load_2d(to + V_ * kPanel, &map, (int)v_col, tok, b);
    }
#pragma unroll
    for (int d = 0; d < DP; ++d) {
      if (warp == ((2 + 2 * d) & 3)) tma_load_2d(to + d * kPanel, &map, (int)q_col + 64 * d, tok, b);
      if (warp == ((3 + 2 * d) & 3)) tma_load_2d(to + (K_ + d) * kPanel, &map, (int)k_col + 64 * d, tok, b);
    }
  };
  if (lane == 0) load_chunk(0);
  if (warp == 0) load_gates(0);
  for (int ch = 0; ch < chunks; ++ch) {
    const int n = min(C, count - ch * C);
    const int64_t tok = t0 + (int64_t)ch * C;
    float* ls = token_values + (ch & 1) * 6 * C;
    float *el = ls + C, *bs = el + C, *zs = bs + C, *rs = zs + C, *es = rs + C;
    unsigned char* cur = panels + (ch & 1) * NB * kPanel;
    if (warp == 0) {
      load_gates(ch + 1);
      cp_async_wait<1>();
      __syncwarp();
      const float4 z = make_float4(0.0f, 0.0f, 0.0f, 0.0f), *src = gs + (ch & 1) * C;
      const float4 ga = lane < n ? src[lane] : z, gb = lane + 32 < n ? src[lane + 32] : z;
      float la = ga.x * 1.4426950408889634f, lb = gb.x * 1.4426950408889634f;
      sum64(la, lb, lane);
      const float last = __shfl_sync(FULL_MASK, lb, 31);
      ls[lane] = la; ls[lane + 32] = lb;
      el[lane] = exp2_fast(la); el[lane + 32] = exp2_fast(lb);
      bs[lane] = ga.y; bs[lane + 32] = gb.y;
      zs[lane] = ga.z; zs[lane + 32] = gb.z;
      rs[lane] = DELTA ? ga.w : p.q_scale; rs[lane + 32] = DELTA ? gb.w : p.q_scale;
      es[lane] = exp2_fast(last - la) * (DELTA ? ga.z : ga.y); es[lane + 32] = exp2_fast(last - lb) * (DELTA ? gb.z : gb.y);
    }
    if (DELTA) async_fence();                              // (the scores were written over the values)
    // every warp is done with the chunk before: its panels may be replaced
    const bool late = !mbar_wait(bar + 8 * (ch & 1), (ch >> 1) & 1, 7);
    if (__syncthreads_or(late)) {                          // expired (the status word says so): once more for the copies, and out
      mbar_wait(bar + 8 * (ch & 1), (ch >> 1) & 1, 7);
      return;
    }
    if (lane == 0) {
      if (DELTA && warp == 0) {
        mbar_expect_tx(bar + 16, 2 * kPanel);
        bulk_copy(p_base + T_ * kPanel, inverse + (chunk_index(t0, seq, ch) * p.heads + h) * (2 * C * C), 2 * kPanel, bar + 16);
      }
      if (ch + 1 < chunks) load_chunk(ch + 1);
    }
    if (n < C) {                                          // behind the portion: k and v of other sequences, to be zero here
      for (int i = tid; i < (C - n) * 8 * (DP + 1); i += THREADS) {
        const int r = n + i / (8 * (DP + 1)), c = i % (8 * (DP + 1));
        *reinterpret_cast<uint4*>(cur + (K_ + (c >> 3)) * kPanel + r * 128 + (c & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
      }
      __syncthreads();
    }

    float u[8][4];                                        // DELTA: U^T
    if (DELTA) {
      bool there = true;
      if (works) {
        float r[8][4] = {};                               // right-hand side beta (v - e^L K S_0), transposed
        state_times(K_, r);
#pragma unroll
        for (int kb = 0; kb < 4; ++kb) {
          unsigned v[4];
          values(kb, v);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int t = kb * 16 + 8 * i + q2;
            const float2 x = bf16x2_to_f32(v[2 * i]), y = bf16x2_to_f32(v[2 * i + 1]);
            const float2 b = *reinterpret_cast<const float2*>(bs + t), e = *reinterpret_cast<const float2*>(el + t), z = *reinterpret_cast<const float2*>(zs + t);
            const float b0 = b.x, b1 = b.y, f0 = e.x * z.x, f1 = e.y * z.y;
            float* a = r[2 * kb + i];
            a[0] = b0 * (x.x - f0 * a[0]); a[1] = b1 * (x.y - f1 * a[1]);
            a[2] = b0 * (y.x - f0 * a[2]); a[3] = b1 * (y.y - f1 * a[3]);
          }
        }
        there = mbar_wait(bar + 16, ch & 1, 7);
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int k = 0; k < 4; ++k) u[i][k] = 0.0f;
#pragma unroll
        for (int kb = 0; kb < 4; ++kb) {
          unsigned ah[4], al[4];
          split2(r[2 * kb][0], r[2 * kb][1], &ah[0], &al[0]);
          split2(r[2 * kb][2], r[2 * kb][3], &ah[1], &al[1]);
          split2(r[2 * kb + 1][0], r[2 * kb + 1][1], &ah[2], &al[2]);
          split2(r[2 * kb + 1][2], r[2 * kb + 1][3], &ah[3], &al[3]);
          unsigned bh[4][4], bl[4][4];
#pragma unroll
          for (int j = kb; j < 4; ++j) {
            mm_ldsm(bh[j], at_fix(T_, j, kb));
            mm_ldsm(bl[j], at_fix(T_ + 1, j, kb));
          }
#pragma unroll
          for (int j = kb; j < 4; ++j) {
            mm_mma(u[2 * j], ah, bh[j][0], bh[j][1]);
            mm_mma(u[2 * j + 1], ah, bh[j][2], bh[j][3]);
          }
#pragma unroll
          for (int j = kb; j < 4; ++j) {
            mm_mma(u[2 * j], al, bh[j][0], bh[j][1]);
            mm_mma(u[2 * j + 1], al, bh[j][2], bh[j][3]);
          }
#pragma unroll
          for (int j = kb; j < 4; ++j) {
            mm_mma(u[2 * j], ah, bl[j][0], bl[j][1]);
            mm_mma(u[2 * j + 1], ah, bl[j][2], bl[j][3]);
          }
        }
      }
      if (__syncthreads_or(!there)) {                     // (the values' place is taken by the scores)
        mbar_wait(bar + 16, ch & 1, 7);
        if (ch + 1 < chunks) mbar_wait(bar + 8 * ((ch + 1) & 1), ((ch + 1) >> 1) & 1, 7);
        return;
      }
    }

    float q_n = 0.0f;                                     // two threads per token: q . n in front of the chunk
    if (with_n) {
      const int t = tid >> 1, half = tid & 1;
      float acc[4] = {};
#pragma unroll
      for (int i = 0; i < DR; ++i) {                      // pieces of 8 values
        if (!FULL && i >= k16) break;
        const int c = 2 * i + half;
        const uint4 x = *reinterpret_cast<const uint4*>(cur + (c >> 3) * kPanel + t * 128 + (((c ^ t) & 7) << 4));
        const float4 n0 = *reinterpret_cast<const float4*>(ns + 8 * c), n1 = *reinterpret_cast<const float4*>(ns + 8 * c + 4);
        const float2 x0 = bf16x2_to_f32(x.x), x1 = bf16x2_to_f32(x.y), x2 = bf16x2_to_f32(x.z), x3 = bf16x2_to_f32(x.w);
        acc[0] = fmaf(x0.x, n0.x, fmaf(x0.y, n0.y, acc[0]));
        acc[1] = fmaf(x1.x, n0.z, fmaf(x1.y, n0.w, acc[1]));
        acc[2] = fmaf(x2.x, n1.x, fmaf(x2.y, n1.y, acc[2]));
        acc[3] = fmaf(x3.x, n1.z, fmaf(x3.y, n1.w, acc[3]));
      }
      q_n = (acc[0] + acc[1]) + (acc[2] + acc[3]);
      q_n += __shfl_xor_sync(FULL_MASK, q_n, 1);
#pragma unroll
      for (int i0 = 0; i0 < 16 * DR; i0 += THREADS) {     // sums of 8 decayed keys, 8 entries of each
        const int i = i0 + tid, pieces = FULL ? 2 * DR : 2 * k16, tg = i / pieces, c = i - tg * pieces;
        if (i >= 16 * k16) break;
        float acc[8] = {};
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const uint4 x = *reinterpret_cast<const uint4*>(cur + (K_ + (c >> 3)) * kPanel + (8 * tg + u) * 128 + (((c ^ u) & 7) << 4));
          const unsigned w[4] = {x.x, x.y, x.z, x.w};
          const float e = es[8 * tg + u];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float2 f = bf16x2_to_f32(w[k]);
            acc[2 * k] = fmaf(e, f.x, acc[2 * k]);
            acc[2 * k + 1] = fmaf(e, f.y, acc[2 * k + 1]);
          }
        }
        float4* dst = reinterpret_cast<float4*>(np + tg * 16 * DR + 8 * c);
        dst[0] = make_float4(acc[0], acc[1], acc[2], acc[3]);
        dst[1] = make_float4(acc[4], acc[5], acc[6], acc[7]);
      }
    }

    // decayed scores: the ten 16 x 16 blocks on and below the diagonal
    constexpr int WARPS = THREADS / 32, MINE = (10 + WARPS - 1) / WARPS;
    float sc[MINE][2][4];
#pragma unroll
    for (int m = 0; m < MINE; ++m)
#pragma unroll
      for (int k = 0; k < 8; ++k) sc[m][k >> 2][k & 3] = 0.0f;
#pragma unroll
    for (int kk = 0; kk < DR; ++kk) {
      if (!FULL && kk >= k16) break;
      unsigned a[MINE][4], b[MINE][4];
#pragma unroll
      for (int m = 0; m < MINE; ++m) {
        const int blk = min(warp + m * WARPS, 9), rb = (blk >= 1) + (blk >= 3) + (blk >= 6), kb = blk - rb * (rb + 1) / 2;
        mm_ldsm(a[m], at_m(0, rb, kk));
        mm_ldsm(b[m], at_n(K_, kb, kk));
      }
#pragma unroll
      for (int m = 0; m < MINE; ++m) {
        mm_mma(sc[m][0], a[m], b[m][0], b[m][1]);
        mm_mma(sc[m][1], a[m], b[m][2], b[m][3]);
      }
    }
#pragma unroll
    for (int m = 0; m < MINE; ++m) {
      const int blk = warp + m * WARPS;
      if (blk >= 10) break;
      const int rb = (blk >= 1) + (blk >= 3) + (blk >= 6), kb = blk - rb * (rb + 1) / 2;
      float (&s)[2][4] = sc[m];
      const int ra = rb * 16 + g;
      const float la = ls[ra], lb = ls[ra + 8];
      float sum_a = 0.0f, sum_b = 0.0f;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int c = kb * 16 + 8 * i + q2;
        const float2 l = *reinterpret_cast<const float2*>(ls + c), w = *reinterpret_cast<const float2*>((DELTA ? zs : bs) + c);
        const float l0 = l.x, l1 = l.y, w0 = w.x, w1 = w.y;
        float s0 = s[i][0] * exp2_fast(la - l0) * w0, s1 = s[i][1] * exp2_fast(la - l1) * w1;
        float s2 = s[i][2] * exp2_fast(lb - l0) * w0, s3 = s[i][3] * exp2_fast(lb - l1) * w1;
        s0 = c <= ra ? s0 : 0.0f;
        s1 = c < ra ? s1 : 0.0f;
        s2 = c <= ra + 8 ? s2 : 0.0f;
        s3 = c < ra + 8 ? s3 : 0.0f;
        sum_a += s0 + s1;
        sum_b += s2 + s3;
        unsigned hi, lo;
        split2(s0, s1, &hi, &lo);
        const int to = ra * 128 + (((kb * 2 + i) ^ g) << 4) + 2 * q2;                  // (row ra + 8 has the same last bits)
        unsigned char *hp = (DELTA ? cur : panels) + PH_ * kPanel + to, *lp = panels + PL_ * kPanel + to;
        *reinterpret_cast<unsigned*>(hp) = hi;
        *reinterpret_cast<unsigned*>(lp) = lo;
        split2(s2, s3, &hi, &lo);
        *reinterpret_cast<unsigned*>(hp + 8 * 128) = hi;
        *reinterpret_cast<unsigned*>(lp + 8 * 128) = lo;
      }
      if (with_n) {
#pragma unroll
        for (int o = 1; o < 4; o <<= 1) {
          sum_a += __shfl_xor_sync(FULL_MASK, sum_a, o);
          sum_b += __shfl_xor_sync(FULL_MASK, sum_b, o);
        }
        if (q2 == 0) {
          nsum[kb * C + ra] = sum_a;
          nsum[kb * C + ra + 8] = sum_b;
        }
      }
    }
    __syncthreads();
    if (with_n) {
      const int t = tid >> 1;
      if ((tid & 1) == 0 && t < n) {
        float dot = q_n * el[t];
#pragma unroll
        for (int kb = 0; kb < 4; ++kb)
          if (kb <= t >> 4) dot += nsum[kb * C + t];
        p.den[(tok + t) * p.heads + h] = fmaxf(fabsf(dot * rs[t]), zs[t]) + kUnitEps;
      }
      for (int d = tid; d < 16 * k16; d += THREADS) {
        float v = ns[d] * el[C - 1];
#pragma unroll
        for (int tg = 0; tg < 8; ++tg) v += np[tg * 16 * DR + d];
        ns[d] = v;
      }
    }

    if (works) {
      float o[8][4] = {};
      state_times(0, o);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float2 e = *reinterpret_cast<const float2*>(el + i * 8 + q2);
        o[i][0] *= e.x; o[i][1] *= e.y; o[i][2] *= e.x; o[i][3] *= e.y;
      }
      const float decay = el[C - 1];
#pragma unroll
      for (int i = 0; i < 2 * DR; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) S[i][k] *= decay;
#pragma unroll
      for (int kb = 0; kb < 4; ++kb) {
        // the written vectors of 16 tokens: bare for the read-outs of this chunk, decayed to its end for the state
        unsigned wh[4], wl[4], dh[4], dl[4];
        const float2 e0 = *reinterpret_cast<const float2*>(es + kb * 16 + q2), e1 = *reinterpret_cast<const float2*>(es + kb * 16 + 8 + q2);
        if (DELTA) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float* x = &u[2 * kb + (i >> 1)][2 * (i & 1)];
            const float2 e = i < 2 ? e0 : e1;
            split2(x[0], x[1], &wh[i], &wl[i]);
            split2(x[0] * e.x, x[1] * e.y, &dh[i], &dl[i]);
          }
        } else {
          values(kb, wh);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float2 x = bf16x2_to_f32(wh[i]), e = i < 2 ? e0 : e1;
            split2(x.x * e.x, x.y * e.y, &dh[i], &dl[i]);
            if (KIND == B200F_MEMORY_SSD) {
              float* y = &o[2 * kb + (i >> 1)][2 * (i & 1)];
              y[0] = fmaf(skip, x.x, y[0]);
              y[1] = fmaf(skip, x.y, y[1]);
            }
          }
        }
        unsigned bh[4][4], bl[4][4];
#pragma unroll
        for (int j = kb; j < 4; ++j) {
          mm_ldsm(bh[j], DELTA ? at_n(PH_, j, kb) : at_fix(PH_, j, kb));
          mm_ldsm(bl[j], at_fix(PL_, j, kb));
        }
#pragma unroll
        for (int j = kb; j < 4; ++j) {
          mm_mma(o[2 * j], wh, bh[j][0], bh[j][1]);
          mm_mma(o[2 * j + 1], wh, bh[j][2], bh[j][3]);
        }
        if (DELTA) {
#pragma unroll
          for (int j = kb; j < 4; ++j) {
            mm_mma(o[2 * j], wl, bh[j][0], bh[j][1]);
            mm_mma(o[2 * j + 1], wl, bh[j][2], bh[j][3]);
          }
        }
#pragma unroll
        for (int j = kb; j < 4; ++j) {
          mm_mma(o[2 * j], wh, bl[j][0], bl[j][1]);
          mm_mma(o[2 * j + 1], wh, bl[j][2], bl[j][3]);
        }
        constexpr int KG = DR < 4 ? DR : 4;
#pragma unroll
        for (int k0 = 0; k0 < DR; k0 += KG) {
          if (!FULL && k0 >= k16) break;
          unsigned b[KG][4];
#pragma unroll
          for (int i = 0; i < KG; ++i) mm_ldsm_t(b[i], at_m(K_, kb, k0 + i));
#pragma unroll
          for (int i = 0; i < KG; ++i) {
            mm_mma(S[2 * (k0 + i)], dh, b[i][0], b[i][1]);
            mm_mma(S[2 * (k0 + i) + 1], dh, b[i][2], b[i][3]);
          }
#pragma unroll
          for (int i = 0; i < KG; ++i) {
            mm_mma(S[2 * (k0 + i)], dl, b[i][0], b[i][1]);
            mm_mma(S[2 * (k0 + i) + 1], dl, b[i][2], b[i][3]);
          }
        }
      }
      {
        const int64_t pitch = (int64_t)p.heads * p.vdim;
        float* out = p.out + (tok + q2) * pitch + (int64_t)h * p.vdim + col0 + c_lo;
        const bool lo = col0 + c_lo < vp, hi = col0 + c_hi < vp;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float2 r = *reinterpret_cast<const float2*>(rs + i * 8 + q2);
          const bool t_a = i * 8 + q2 < n, t_b = i * 8 + q2 + 1 < n;
          if (t_a && lo) out[0] = o[i][0] * r.x;
          if (t_b && lo) out[pitch] = o[i][1] * r.y;
          if (t_a && hi) out[8] = o[i][2] * r.x;
          if (t_b && hi) out[pitch + 8] = o[i][3] * r.y;
          out += 8 * pitch;
        }
      }
    }
    const unsigned other = ch & 1 ? 0u - NB * kPanel : NB * kPanel;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      n_at[i] += other;
      m_at[i] += other;
    }
    v_at += other;
  }
  __syncthreads();
  if (with_n)
    for (int d = tid; d < p.dim; d += THREADS) nst[d] = ns[d];
  if (!works) return;
#pragma unroll
  for (int i = 0; i < 2 * DR; ++i)
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int d = i * 8 + q2 + (k & 1), c = k < 2 ? c_lo : c_hi;
      if (!FULL && d >= p.dim) continue;
      if (col0 + c < vp) st[(int64_t)d * vp + c] = S[i][k];
    }
}

// (I + M)^-1 of every chunk and head, as two bf16 panels (the 16 x 16 blocks above the diagonal are left undefined), and the
// unit factors of k and q into the gates.  A CTA of 4 warps per (chunk, q / k head); k . k on the tensor cores once, then head
// by head: M, the inverses D_i of its four diagonal blocks by substitution, and the blocks below them column by column from
// T_ij = -D_i sum_(j <= k < i) M_ik T_kj.  The products are transposed as in the chunk kernel, so a block goes from
// accumulator to left operand in registers; operands are two bf16 numbers each.
__global__ void __launch_bounds__(128, 5)
delta_inverse_kernel(const MemoryParams p, const bf16* __restrict__ rows, bf16* __restrict__ inverse) {
  extern __shared__ __align__(128) unsigned char smem[];
  constexpr int C = kChunk;
  const int lk = ((p.dim + 15) & ~15) + 8, k16 = (p.dim + 15) >> 4;
  float* dg = reinterpret_cast<float*>(smem);            // [4][16][16] diagonal blocks of M
  float *ls = dg + 4 * 256, *bs = ls + C, *rk = bs + C, *rq = rk + C;                 // [C] each
  unsigned char *mp = reinterpret_cast<unsigned char*>(rq + C), *tp = mp + 2 * kPanel; // M and the inverse: a high and a low panel each
  bf16* ks = reinterpret_cast<bf16*>(tp);                // [C][lk] keys, until their products are there
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, q2 = 2 * (lane & 3);
  const int ch = blockIdx.x, qh = blockIdx.y, seq = blockIdx.z;
  const int64_t t0 = p.seq_start[seq];
  const int count = p.seq_start[seq + 1] - (int)t0;
  if (ch * C >= count) return;
  const int n = min(C, count - ch * C), cq = p.dim / 8, per = p.heads / p.qk_heads;
  const int64_t tok = t0 + (int64_t)ch * C;
  const bf16* q_src = rows + tok * p.row_pitch + p.q_off + (int64_t)qh * p.dim;
  const bf16* k_src = rows + tok * p.row_pitch + p.k_off + (int64_t)qh * p.dim;
  for (int i = tid; i < C * cq; i += 128) {
    const int t = i / cq, c = (i - t * cq) * 8;
    cp_async16_or_zero(smem_u32(ks + t * lk + c), k_src + (t < n ? t : 0) * p.row_pitch + c, t < n);
  }
  cp_async_commit();
  for (int r = tid; r < C; r += 128)
    for (int c = p.dim; c < lk; ++c) ks[r * lk + c] = __float2bfloat16_rn(0.0f);
  {                                                      // two threads per token
    const int t = tid >> 1;
    const int64_t off = (int64_t)(t < n ? t : 0) * p.row_pitch + (tid & 1) * (p.dim / 2);
    const uint4 *qp = reinterpret_cast<const uint4*>(q_src + off), *kp = reinterpret_cast<const uint4*>(k_src + off);
    auto squares = [](const uint4& v) {
      const unsigned w[4] = {v.x, v.y, v.z, v.w};
      float ss = 0.0f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 x = bf16x2_to_f32(w[k]);
        ss = fmaf(x.x, x.x, fmaf(x.y, x.y, ss));
      }
      return ss;
    };
    float sq = 0.0f, sk = 0.0f;
#pragma unroll 4
    for (int c = 0; c < p.dim / 16; ++c) {
      sq += squares(__ldg(qp + c));
      sk += squares(__ldg(kp + c));
    }
    sq += __shfl_xor_sync(FULL_MASK, sq, 1);
    sk += __shfl_xor_sync(FULL_MASK, sk, 1);
    if ((tid & 1) == 0) {
      rq[t] = p.q_scale / sqrtf(sq + kUnitEps);
      rk[t] = 1.0f / sqrtf(sk + kUnitEps);
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  float gm[4][2][4];                                     // this warp's 16 rows of k . k
#pragma unroll
  for (int kb = 0; kb < 4; ++kb) {
    if (kb > warp) break;
#pragma unroll
    for (int i = 0; i < 8; ++i) gm[kb][i >> 2][i & 3] = 0.0f;
    for (int kk = 0; kk < k16; ++kk) {
      unsigned a[4], b[4];
      mm_ldsm(a, smem_u32(ks + (warp * 16 + (lane & 15)) * lk + (lane >> 4) * 8 + kk * 16));
      mm_ldsm(b, smem_u32(ks + (kb * 16 + (lane & 7) + ((lane >> 4) << 3)) * lk + ((lane >> 3) & 1) * 8 + kk * 16));
      mm_mma(gm[kb][0], a, b[0], b[1]);
      mm_mma(gm[kb][1], a, b[2], b[3]);
    }
  }
  const unsigned m_base = smem_u32(mp), t_base = smem_u32(tp);
  const unsigned n_row = ((lane & 7) + ((lane >> 4) << 3)) * 128, n_x = (((lane >> 3) & 1) ^ (lane & 7)) << 4;
  auto at_n = [&](unsigned base, int row16, int col16) { return base + row16 * 2048 + n_row + (n_x ^ (col16 << 5)); };
  // d [16, 16] += (ah + al) (b_high + b_low) for a right operand stored [n][k] in block (row16, col16) of a pair of panels
  auto times = [&](float (&d)[2][4], const unsigned (&ah)[4], const unsigned (&al)[4], unsigned base, int row16, int col16) {
    unsigned bh[4], bl[4];
    mm_ldsm(bh, at_n(base, row16, col16));
    mm_ldsm(bl, at_n(base + kPanel, row16, col16));
    mm_mma(d[0], ah, bh[0], bh[1]);
    mm_mma(d[1], ah, bh[2], bh[3]);
    mm_mma(d[0], al, bh[0], bh[1]);
    mm_mma(d[1], al, bh[2], bh[3]);
    mm_mma(d[0], ah, bl[0], bl[1]);
    mm_mma(d[1], ah, bl[2], bl[3]);
  };
  for (int e = 0; e < per; ++e) {
    const int h = qh * per + e;
    if (warp == 0) {
      const float4 z = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      float4* gp = p.gates + (tok + lane) * p.heads + h;
      const float4 ga = lane < n ? gp[0] : z, gb = lane + 32 < n ? gp[(int64_t)32 * p.heads] : z;
      float a = ga.x * 1.4426950408889634f, b = gb.x * 1.4426950408889634f;
      sum64(a, b, lane);
      ls[lane] = a; ls[lane + 32] = b;
      bs[lane] = ga.y; bs[lane + 32] = gb.y;
      if (lane < n) { gp[0].z = rk[lane]; gp[0].w = rq[lane]; }
      if (lane + 32 < n) { gp[(int64_t)32 * p.heads].z = rk[lane + 32]; gp[(int64_t)32 * p.heads].w = rq[lane + 32]; }
    }
    __syncthreads();
    const int ra = warp * 16 + g;
    const float la = ls[ra], lb = ls[ra + 8], fa = bs[ra] * rk[ra], fb = bs[ra + 8] * rk[ra + 8];
#pragma unroll
    for (int kb = 0; kb < 4; ++kb) {
      if (kb > warp) break;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int c = kb * 16 + 8 * i + q2;
        const float2 l = *reinterpret_cast<const float2*>(ls + c), r = *reinterpret_cast<const float2*>(rk + c);
        const float (&s)[4] = gm[kb][i];
        float s0 = s[0] * fa * r.x * exp2_fast(la - l.x), s1 = s[1] * fa * r.y * exp2_fast(la - l.y);
        float s2 = s[2] * fb * r.x * exp2_fast(lb - l.x), s3 = s[3] * fb * r.y * exp2_fast(lb - l.y);
        if (kb < warp) {
          unsigned hi, lo;
          unsigned char* at = mp + ra * 128 + (((kb * 2 + i) ^ g) << 4) + 2 * q2;       // (row ra + 8 has the same last bits)
          split2(s0, s1, &hi, &lo);
          *reinterpret_cast<unsigned*>(at) = hi;
          *reinterpret_cast<unsigned*>(at + kPanel) = lo;
          split2(s2, s3, &hi, &lo);
          *reinterpret_cast<unsigned*>(at + 8 * 128) = hi;
          *reinterpret_cast<unsigned*>(at + 8 * 128 + kPanel) = lo;
        } else {
          float* at = dg + kb * 256 + g * 16 + 8 * i + q2;                              // entries above the diagonal are not read
          *reinterpret_cast<float2*>(at) = make_float2(s0, s1);
          *reinterpret_cast<float2*>(at + 128) = make_float2(s2, s3);
        }
      }
    }
    __syncthreads();
    if (tid < C) {                                       // column c of a diagonal block's inverse
      const int b = tid >> 4, c = tid & 15;
      const float* m = dg + b * 256;
      float x[16];
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        float a0 = t == c ? 1.0f : 0.0f, a1 = 0.0f;
#pragma unroll
        for (int s = 0; s < t; s += 2) {
          const float2 v = *reinterpret_cast<const float2*>(m + t * 16 + s);
          a0 = fmaf(-v.x, x[s], a0);
          if (s + 1 < t) a1 = fmaf(-v.y, x[s + 1], a1);
        }
        x[t] = a0 + a1;
        const bf16 hi = __float2bfloat16_rn(x[t]);
        bf16* at = reinterpret_cast<bf16*>(tp + panel_at(b * 16 + t, b * 16 + c));
        at[0] = hi;
        at[C * C] = __float2bfloat16_rn(x[t] - __bfloat162float(hi));
      }
    }
    __syncthreads();
    if (warp < 3) {                                      // block column `warp`
      unsigned th[3][4], tl[3][4];                       // T_kj transposed, as left operands
      mm_ldsm_t(th[0], at_n(t_base, warp, warp));
      mm_ldsm_t(tl[0], at_n(t_base + kPanel, warp, warp));
#pragma unroll
      for (int d = 1; d < 4; ++d) {
        const int i = warp + d;
        if (i >= 4) break;
        float x[2][4] = {}, y[2][4] = {};
#pragma unroll
        for (int k = 0; k < d; ++k) times(x, th[k], tl[k], m_base, i, warp + k);
        unsigned xh[4], xl[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) split2(-x[k >> 1][2 * (k & 1)], -x[k >> 1][2 * (k & 1) + 1], &xh[k], &xl[k]);
        times(y, xh, xl, t_base, i, i);
        unsigned yh[4], yl[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          split2(y[k >> 1][2 * (k & 1)], y[k >> 1][2 * (k & 1) + 1], &yh[k], &yl[k]);
          // rows of T: 8 (k >> 1) + q2 and the next; column: g + 8 (k & 1)
          const int row = i * 16 + 8 * (k >> 1) + q2, col = warp * 16 + g + 8 * (k & 1);
          *reinterpret_cast<unsigned short*>(tp + panel_at(row, col)) = (unsigned short)yh[k];
          *reinterpret_cast<unsigned short*>(tp + panel_at(row + 1, col)) = (unsigned short)(yh[k] >> 16);
          *reinterpret_cast<unsigned short*>(tp + kPanel + panel_at(row, col)) = (unsigned short)yl[k];
          *reinterpret_cast<unsigned short*>(tp + kPanel + panel_at(row + 1, col)) = (unsigned short)(yl[k] >> 16);
        }
        if (d < 3) {
#pragma unroll
          for (int k = 0; k < 4; ++k) { th[d][k] = yh[k]; tl[d][k] = yl[k]; }
        }
      }
    }
    __syncthreads();
    uint4* dst = reinterpret_cast<uint4*>(inverse + (chunk_index(t0, seq, ch) * p.heads + h) * (2 * C * C));
#pragma unroll
    for (int i = 0; i < 2 * kPanel / 16 / 128; ++i) dst[tid + 128 * i] = *reinterpret_cast<const uint4*>(tp + (tid + 128 * i) * 16);
    __syncthreads();                                     // the panels may be replaced
  }
}

// ---------------------------------------------------------------------------------------------------
// Decode: a CTA per (sequence, head, slice of VQ column quads); 256 / VQ row groups, R rows per thread in registers.
template <typename T, int KIND, int R>
__global__ void __launch_bounds__(256)
memory_step_kernel(const MemoryParams p, const T* __restrict__ rows, int vq) {
  __shared__ float qs[512], ks[512], scratch[32];
  __shared__ float4 red[256];
  pdl_launch_dependents();
  const int tid = threadIdx.x, tx = tid % vq, ty = tid / vq, rg = 256 / vq;
  const int slice = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int vp = pad8i(p.vdim), hq = pad8i(p.dim), c = (slice * vq + tx) * 4;
  const int qh = h / (p.heads / p.qk_heads);
  pdl_wait();
  const int64_t slot_head = (int64_t)p.slots[seq] * p.heads + h;
  const bool has_state = p.positions[seq] > 0;
  float* st = p.state + slot_head * p.dim * vp + c;
  float4 S[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int n = ty + i * rg;
    S[i] = (has_state && n < p.dim && c < vp) ? __ldcs(reinterpret_cast<const float4*>(st + (int64_t)n * vp)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  const T* row = rows + (int64_t)seq * p.row_pitch;
  float sq = 0.0f, sk = 0.0f;
  for (int i = tid; i < rg * R; i += 256) {
    const float q = i < p.dim ? to_f32(row[p.q_off + (int64_t)qh * hq + i]) : 0.0f, k = i < p.dim ? to_f32(row[p.k_off + (int64_t)qh * hq + i]) : 0.0f;
    qs[i] = q;
    ks[i] = k;
    sq = fmaf(q, q, sq);
    sk = fmaf(k, k, sk);
  }
  float4 g = p.gates[(int64_t)seq * p.heads + h];
  g.x = expf(g.x);
  g.w = p.q_scale;
  if (KIND == B200F_MEMORY_DELTA) {
    g.w = p.q_scale / sqrtf(block_sum(sq, scratch) + kUnitEps);
    g.z = 1.0f / sqrtf(block_sum(sk, scratch) + kUnitEps);
  }
  float v[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) v[k] = c + k < p.vdim ? to_f32(row[p.v_off + (int64_t)h * vp + c + k]) : 0.0f;
  __syncthreads();
  if (KIND == B200F_MEMORY_EXP && slice == 0) {
    float* nst = p.norm_state + slot_head * (p.dim + 1);
    float dot = 0.0f;
    for (int i = tid; i < p.dim; i += 256) {
      const float n = fmaf(g.y, ks[i], g.x * (has_state ? nst[i] : 0.0f));
      nst[i] = n;
      dot = fmaf(n, qs[i], dot);
    }
    dot = block_sum(dot, scratch) * p.q_scale;
    if (tid == 0) p.den[(int64_t)seq * p.heads + h] = fmaxf(fabsf(dot), g.z) + kUnitEps;
  }
  // sums over the row groups, for every thread of a column
  auto total = [&](float4 mine) {
    __syncthreads();
    red[tid] = mine;
    __syncthreads();
    float4 r = red[tx];
    for (int i = 1; i < rg; ++i) {
      const float4 o = red[i * vq + tx];
      r.x += o.x; r.y += o.y; r.z += o.z; r.w += o.w;
    }
    return r;
  };
  float w[4] = {g.y * v[0], g.y * v[1], g.y * v[2], g.y * v[3]};
  if (KIND == B200F_MEMORY_DELTA) {
    float4 d = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const float k = ks[ty + i * rg];
      d.x = fmaf(S[i].x, k, d.x); d.y = fmaf(S[i].y, k, d.y); d.z = fmaf(S[i].z, k, d.z); d.w = fmaf(S[i].w, k, d.w);
    }
    d = total(d);
    const float f = g.y * g.x * g.z;
    w[0] = (w[0] - f * d.x) * g.z; w[1] = (w[1] - f * d.y) * g.z; w[2] = (w[2] - f * d.z) * g.z; w[3] = (w[3] - f * d.w) * g.z;
  }
  float4 o = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int n = ty + i * rg;
    const float k = ks[n], q = qs[n];
    S[i].x = fmaf(k, w[0], g.x * S[i].x); S[i].y = fmaf(k, w[1], g.x * S[i].y);
    S[i].z = fmaf(k, w[2], g.x * S[i].z); S[i].w = fmaf(k, w[3], g.x * S[i].w);
    o.x = fmaf(S[i].x, q, o.x); o.y = fmaf(S[i].y, q, o.y); o.z = fmaf(S[i].z, q, o.z); o.w = fmaf(S[i].w, q, o.w);
    if (n < p.dim && c < vp) __stcs(reinterpret_cast<float4*>(st + (int64_t)n * vp), S[i]);
  }
  o = total(o);
  if (ty == 0) {
    const float skip = p.skip ? p.skip[h] : 0.0f;
    const float r[4] = {fmaf(skip, v[0], o.x * g.w), fmaf(skip, v[1], o.y * g.w), fmaf(skip, v[2], o.z * g.w), fmaf(skip, v[3], o.w * g.w)};
    float* dst = p.out + ((int64_t)seq * p.heads + h) * p.vdim + c;
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (c + k < p.vdim) dst[k] = r[k];
  }
}

// ---------------------------------------------------------------------------------------------------
struct MemoryOutput {
  const float *o, *den;                // den nullable: [rows][heads]
  int heads, vdim, group;              // group: values per norm
  const float* y;                      // parts that hold the gate's projection
  int splits;
  int64_t split_stride, y_pitch, gate_col;
  int gate;                            // B200F_GATE_*
  const float* norm_w;
  int norm_len;                        // entry i of a row has gain norm_w[i % norm_len]
  float eps;
  int64_t out_pitch;
  int64_t rows;
  int wpg, cta_rows;                   // warps per group, rows per CTA
};

// A CTA per row, or per several short ones.  A warp per group, or several for the wide groups of a few; up to kOutKeep packs of a group per lane stay in
// registers between the sum of squares and the result, the others are formed twice.
constexpr int kOutKeep = 2;
template <int V>
struct alignas(4 * V) OutPack { float v[V]; };

template <typename T, int V>
__global__ void __launch_bounds__(256, 4)
memory_output_kernel(const MemoryOutput p, T* __restrict__ out) {
  __shared__ float part[8];
  pdl_launch_dependents();
  pdl_wait();
  const int n = p.heads * p.vdim, groups = n / p.group;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wpg = p.wpg, at_once = 8 / wpg, sub = warp % wpg;                  // warps per group
  const int64_t row0 = (int64_t)blockIdx.x * p.cta_rows;
  const int units = (int)min((int64_t)p.cta_rows, p.rows - row0) * groups;     // (row, group) pairs of this CTA
  const int step = 32 * wpg * V;
  auto load = [&](const float* src) { return *reinterpret_cast<const OutPack<V>*>(src); };
  const float *o = nullptr, *gate = nullptr;
  auto gate_at = [&](int c) {
    OutPack<V> z = load(gate + c);
    for (int s = 1; s < p.splits; ++s) {
      const OutPack<V> x = load(gate + c + s * p.split_stride);
#pragma unroll
      for (int k = 0; k < V; ++k) z.v[k] += x.v[k];
    }
    return z;
  };
  for (int u0 = 0; u0 < units; u0 += at_once) {
    const int unit = u0 + warp / wpg;
    const bool live = warp / wpg < at_once && unit < units;
    const int r = live ? unit / groups : 0, g = live ? unit - r * groups : 0, c0 = g * p.group;
    const int64_t row = row0 + r;
    o = p.o + row * n;
    gate = p.y + row * p.y_pitch + p.gate_col;
    const float inv_den = live && p.den ? 1.0f / p.den[row * p.heads + g] : 1.0f;         // with den a group is a head
    auto value = [&](int i) {
      OutPack<V> u = load(o + c0 + i);
      if (p.gate == B200F_GATE_SILU_BEFORE) {
        const OutPack<V> z = gate_at(c0 + i);
#pragma unroll
        for (int k = 0; k < V; ++k) u.v[k] *= silu_f32(z.v[k]);
      }
      return u;
    };
    OutPack<V> keep[kOutKeep], z[kOutKeep];
    float ss = 0.0f;
    const int first = (sub * 32 + lane) * V;
#pragma unroll
    for (int j = 0; j < kOutKeep; ++j) {
      const int i = first + j * step;
      if (live && i < p.group) {
        keep[j] = value(i);
        if (p.gate != B200F_GATE_SILU_BEFORE) z[j] = gate_at(c0 + i);
#pragma unroll
        for (int k = 0; k < V; ++k) ss = fmaf(keep[j].v[k], keep[j].v[k], ss);
      }
    }
    if (live)
      for (int i = first + kOutKeep * step; i < p.group; i += step) {
        const OutPack<V> u = value(i);
#pragma unroll
        for (int k = 0; k < V; ++k) ss = fmaf(u.v[k], u.v[k], ss);
      }
    ss = warp_sum(ss);
    if (wpg > 1) {
      if (lane == 0) part[warp] = ss;
      __syncthreads();
      ss = 0.0f;
      for (int i = 0; i < wpg; ++i) ss += live ? part[(warp / wpg) * wpg + i] : 0.0f;
      __syncthreads();
    }
    if (!live) continue;
    const float inv = inv_den / sqrtf(ss * inv_den * inv_den / (float)p.group + p.eps);
    const float* w = p.norm_w + (p.norm_len == n ? c0 : 0);
    T* dst = out + row * p.out_pitch + c0;
    auto finish = [&](int i, const OutPack<V>& u, const OutPack<V>& zz) {
      const OutPack<V> gain = load(w + i);
      OutPack<V> r;
#pragma unroll
      for (int k = 0; k < V; ++k) {
        r.v[k] = u.v[k] * inv * gain.v[k];
        if (p.gate != B200F_GATE_SILU_BEFORE) r.v[k] *= p.gate == B200F_GATE_SIGMOID_AFTER ? sigmoid_f32(zz.v[k]) : silu_f32(zz.v[k]);
      }
      if (V == 4) store4(dst + i, make_float4(r.v[0], r.v[V > 1 ? 1 : 0], r.v[V > 2 ? 2 : 0], r.v[V > 3 ? 3 : 0]));
      else
#pragma unroll
        for (int k = 0; k < V; ++k) dst[i + k] = from_f32<T>(r.v[k]);
    };
#pragma unroll
    for (int j = 0; j < kOutKeep; ++j)
      if (first + j * step < p.group) finish(first + j * step, keep[j], z[j]);
    for (int i = first + kOutKeep * step; i < p.group; i += step) finish(i, value(i), p.gate != B200F_GATE_SILU_BEFORE ? gate_at(c0 + i) : z[0]);
  }
}

// ----------------------------------------------------------------------------- host side
template <typename T, int VEC>
static void launch_prepare_taps(const MemoryPrepare& p, T* out, dim3 grid, cudaStream_t st) {
  switch (p.taps) {
    case 0: launch_pdl(memory_prepare_kernel<T, VEC, 0>, grid, dim3(256), 0, st, p, out); break;
    case 2: launch_pdl(memory_prepare_kernel<T, VEC, 2>, grid, dim3(256), 0, st, p, out); break;
    case 3: launch_pdl(memory_prepare_kernel<T, VEC, 3>, grid, dim3(256), 0, st, p, out); break;
    case 4: launch_pdl(memory_prepare_kernel<T, VEC, 4>, grid, dim3(256), 0, st, p, out); break;
    default: launch_pdl(memory_prepare_kernel<T, VEC, -1>, grid, dim3(256), 0, st, p, out); break;
  }
}
template <typename T>
static int launch_prepare(MemoryPrepare p, T* out, int batch, cudaStream_t st) {
  bool vec = p.channels % 4 == 0 && p.y_pitch % 4 == 0 && p.col0 % 4 == 0 && p.split_stride % 4 == 0 && p.out_pitch % 4 == 0 && aligned16(p.y) && aligned16(out);
  for (int s = 0; s < 3; ++s) vec = vec && p.seg_head[s] % 4 == 0;
  const int per = 256 * (vec ? 4 : 1);
  // prompts: enough tokens per thread that re-reading the taps in front of a block is cheap, as long as the GPU stays full
  p.channel_blocks = (p.channels + per - 1) / per;
  p.block_tokens = 1;
  if (p.seq_start)
    while (p.block_tokens < 16 && p.channel_blocks * (p.tokens / (2 * p.block_tokens)) >= 4 * sm_count()) p.block_tokens *= 2;
  while ((p.tokens + p.block_tokens - 1) / p.block_tokens > 65535) p.block_tokens *= 2;
  const int gate_blocks = (p.block_tokens * p.heads + 255) / 256;
  const dim3 grid((unsigned)(p.channel_blocks + gate_blocks), (unsigned)((p.tokens + p.block_tokens - 1) / p.block_tokens));
  if (vec) launch_prepare_taps<T, 4>(p, out, grid, st);
  else launch_prepare_taps<T, 1>(p, out, grid, st);
  int rc = check_launch("memory_prepare");
  if (rc != B200_OK || !p.seq_start) return rc;
  if (p.taps > 1) {
    launch_pdl(conv_state_kernel, dim3((unsigned)((p.channels + 255) / 256), (unsigned)batch), dim3(256), 0, st, p);
    rc = check_launch("memory_prepare (convolution state)");
  }
  if (rc == B200_OK && p.kind == B200F_MEMORY_EXP) {
    launch_pdl(running_max_kernel, dim3((unsigned)p.heads, (unsigned)batch), dim3(32), 0, st, p);
    rc = check_launch("memory_prepare (running maximum)");
  }
  return rc;
}

template <typename T, int KIND, int LN, int R>
static int launch_scan_shape(MemoryParams p, const T* rows, int batch, cudaStream_t st) {
  constexpr int CPW = (32 / LN) * 4;
  const int vp = (p.vdim + 7) & ~7;
  int warps = (vp + CPW - 1) / CPW;
  warps = warps > 8 ? 8 : warps;
  while (warps > 2 && CPW * (warps / 2) % 8 == 0 && (int64_t)((vp + CPW * warps - 1) / (CPW * warps)) * p.heads * batch < 2 * sm_count()) warps = (warps + 1) / 2;
  if (CPW == 4 && warps % 2) ++warps;                        // slices start at multiples of 8 columns
  p.warps = warps;
  const int vs = CPW * warps;
  const size_t bytes = ScanShape<T>(LN * R, p.dim, vs).bytes();
  cudaError_t e = cudaFuncSetAttribute(memory_scan_kernel<T, KIND, LN, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "memory_scan: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  const dim3 grid((unsigned)((vp + vs - 1) / vs), (unsigned)p.heads, (unsigned)batch);
  launch_pdl(memory_scan_kernel<T, KIND, LN, R>, grid, dim3(32 * warps + (KIND == B200F_MEMORY_EXP ? 32 : 0)), bytes, st, p, rows);
  return check_launch("memory_scan");
}
template <int KIND, int DR, bool FULL>
static int launch_chunk_shape(const CUtensorMap& map, const MemoryParams& p, const bf16* inverse, int batch, cudaStream_t st) {
  constexpr size_t need = chunk_smem(DR, KIND), alone = 116 * 1024;
  static_assert(need <= 227 * 1024, "shared memory budget");
  // few CTAs spread over the SMs (launched while the kernel before still runs, two would share one that is free early)
  const int64_t ctas = (int64_t)((p.vdim + kChunkCols - 1) / kChunkCols) * p.heads * batch;
  const size_t bytes = need < alone && ctas <= sm_count() ? alone : need;
  cudaError_t e = cudaFuncSetAttribute(memory_chunk_kernel<KIND, DR, FULL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "memory_scan: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  const dim3 grid((unsigned)((p.vdim + kChunkCols - 1) / kChunkCols), (unsigned)p.heads, (unsigned)batch);
  launch_pdl(memory_chunk_kernel<KIND, DR, FULL>, grid, dim3(kChunkWarps * 32), bytes, st, map, p, inverse);
  return check_launch("memory_scan (chunks)");
}
template <int KIND>
static int launch_chunks(const MemoryParams& p, const bf16* rows, bf16* inverse, int64_t tokens, int batch, int max_q, cudaStream_t st) {
  CUtensorMap map;
  {
    EncodeTiledFn fn = encode_fn();
    const cuuint64_t dims[2] = {(cuuint64_t)p.row_pitch, (cuuint64_t)tokens};
    const cuuint64_t strides[1] = {(cuuint64_t)p.row_pitch * 2};
    const cuuint32_t box[2] = {64, (cuuint32_t)kChunk}, estr[2] = {1, 1};
    B200_REQUIRE(fn && fn(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16*>(rows), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS,
                 B200_E_CUDA, "memory_scan: cuTensorMapEncodeTiled failed");
  }
  if (KIND == B200F_MEMORY_DELTA) {
    const size_t keys = (size_t)kChunk * (((p.dim + 15) & ~15) + 8) * 2;
    const size_t bytes = (size_t)2 * kPanel + 4 * 256 * 4 + 4 * kChunk * 4 + (keys > 2 * kPanel ? keys : 2 * kPanel);
    cudaError_t e = cudaFuncSetAttribute(delta_inverse_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "memory_scan: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
    launch_pdl(delta_inverse_kernel, dim3((unsigned)((max_q + kChunk - 1) / kChunk), (unsigned)p.qk_heads, (unsigned)batch), dim3(128), bytes, st, p, rows, inverse);
    const int rc = check_launch("memory_scan (inverse)");
    if (rc != B200_OK) return rc;
  }
  if (p.dim == 32) return launch_chunk_shape<KIND, 2, true>(map, p, inverse, batch, st);
  if (p.dim < 32) return launch_chunk_shape<KIND, 2, false>(map, p, inverse, batch, st);
  if (p.dim == 64) return launch_chunk_shape<KIND, 4, true>(map, p, inverse, batch, st);
  if (p.dim < 64) return launch_chunk_shape<KIND, 4, false>(map, p, inverse, batch, st);
  if (p.dim == 128) return launch_chunk_shape<KIND, 8, true>(map, p, inverse, batch, st);
  if (p.dim < 128) return launch_chunk_shape<KIND, 8, false>(map, p, inverse, batch, st);
  return p.dim == 256 ? launch_chunk_shape<KIND, 16, true>(map, p, inverse, batch, st) : launch_chunk_shape<KIND, 16, false>(map, p, inverse, batch, st);
}
// The chunk form: bf16 heads of whole 16-value pieces (q, k) and without padding (v), and portions that fill a good part of a chunk.
static bool chunks_fit(int dtype, int dim, int vdim, int max_q) { return dtype == B200F_BF16 && dim <= 256 && dim % 16 == 0 && vdim % 8 == 0 && max_q > 16; }

template <typename T, int KIND>
static int launch_scan(const MemoryParams& p, const T* rows, int batch, cudaStream_t st) {
  if (p.seq_start) {
    if (p.dim <= 32) return launch_scan_shape<T, KIND, 4, 8>(p, rows, batch, st);
    if (p.dim <= 64) return launch_scan_shape<T, KIND, 8, 8>(p, rows, batch, st);
    if (p.dim <= 128) return launch_scan_shape<T, KIND, 16, 8>(p, rows, batch, st);
    if (p.dim <= 256) return launch_scan_shape<T, KIND, 16, 16>(p, rows, batch, st);
    return launch_scan_shape<T, KIND, 32, 16>(p, rows, batch, st);
  }
  const int vp = (p.vdim + 7) & ~7;
  int vq = 2;
  while (vq < 32 && vq * 4 < vp) vq *= 2;
  while (vq > 2 && (p.dim + 256 / vq - 1) / (256 / vq) > 32) vq /= 2;
  const int r = (p.dim + 256 / vq - 1) / (256 / vq);
  const dim3 grid((unsigned)((vp + 4 * vq - 1) / (4 * vq)), (unsigned)p.heads, (unsigned)batch);
  if (r <= 4) launch_pdl(memory_step_kernel<T, KIND, 4>, grid, dim3(256), 0, st, p, rows, vq);
  else if (r <= 8) launch_pdl(memory_step_kernel<T, KIND, 8>, grid, dim3(256), 0, st, p, rows, vq);
  else if (r <= 16) launch_pdl(memory_step_kernel<T, KIND, 16>, grid, dim3(256), 0, st, p, rows, vq);
  else launch_pdl(memory_step_kernel<T, KIND, 32>, grid, dim3(256), 0, st, p, rows, vq);
  return check_launch("memory_step");
}
template <typename T>
static int launch_memory(const MemoryParams& p, int kind, const T* rows, int batch, cudaStream_t st) {
  switch (kind) {
    case B200F_MEMORY_EXP: return launch_scan<T, B200F_MEMORY_EXP>(p, rows, batch, st);
    case B200F_MEMORY_SSD: return launch_scan<T, B200F_MEMORY_SSD>(p, rows, batch, st);
    default: return launch_scan<T, B200F_MEMORY_DELTA>(p, rows, batch, st);
  }
}
static bool valid_kind(int k) { return k == B200F_MEMORY_EXP || k == B200F_MEMORY_SSD || k == B200F_MEMORY_DELTA; }

}  // namespace b200

using namespace b200;

extern "C" int b200f_memory_prepare(const float* y, int splits, int64_t split_stride, int64_t y_pitch, int64_t col0,
                                    const int32_t* segments, const float* conv_w, const float* conv_b, int taps,
                                    float* conv_state, const int32_t* slots, const int32_t* positions,
                                    const int32_t* seq_start, const int32_t* seq_ids, void* out, int64_t out_pitch, int dtype,
                                    int kind, int heads, int64_t gate_col_a, int64_t gate_col_b, const float* gate_a,
                                    const float* gate_b, float cap, float* gates, float* norm_state, int norm_dim,
                                    int64_t tokens, int batch, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype) && valid_kind(kind), B200_E_UNSUPPORTED, "memory_prepare: dtype %d, kind %d", dtype, kind);
  B200_REQUIRE(segments, B200_E_NULL, "memory_prepare: null pointer");
  MemoryPrepare p{};
  int64_t width = 0, padded = 0;
  for (int i = 0; i < 3; ++i) {
    p.seg_width[i] = segments[2 * i];
    p.seg_head[i] = segments[2 * i + 1];
    B200_REQUIRE(p.seg_width[i] > 0 && p.seg_head[i] > 0 && p.seg_width[i] % p.seg_head[i] == 0, B200_E_SHAPE,
                 "memory_prepare: segment %d has %d columns in heads of %d", i, p.seg_width[i], p.seg_head[i]);
    width += p.seg_width[i];
    padded += (int64_t)(p.seg_width[i] / p.seg_head[i]) * ((p.seg_head[i] + 7) & ~7);
  }
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && batch >= 0 && batch < 65536 && splits >= 1 && width < (1 << 30) && taps >= 0 && heads > 0 &&
                   col0 >= 0 && col0 + width <= y_pitch && out_pitch >= padded && gate_col_a >= 0 && gate_col_a + heads <= y_pitch &&
                   gate_col_b >= 0 && gate_col_b + heads <= y_pitch && (seq_start || tokens == batch) && (kind != B200F_MEMORY_EXP || (norm_dim > 0 && cap > 0)),
               B200_E_SHAPE, "memory_prepare: tokens=%lld batch=%d columns=%lld taps=%d heads=%d", (long long)tokens, batch, (long long)width, taps, heads);
  if (tokens == 0 || batch == 0) return B200_OK;
  B200_REQUIRE(y && slots && positions && out && gates && gate_a && gate_b && (taps == 0 || conv_w) && (taps <= 1 || conv_state) &&
                   (!seq_start == !seq_ids) && (kind != B200F_MEMORY_EXP || norm_state), B200_E_NULL, "memory_prepare: null pointer");
  p.y = y; p.splits = splits; p.split_stride = split_stride; p.y_pitch = y_pitch; p.col0 = col0; p.channels = (int)width;
  p.conv_w = conv_w; p.conv_b = conv_b; p.taps = taps; p.conv_state = conv_state;
  p.slots = slots; p.positions = positions; p.seq_start = seq_start; p.seq_ids = seq_ids; p.out_pitch = out_pitch;
  p.kind = kind; p.heads = heads; p.gate_col_a = gate_col_a; p.gate_col_b = gate_col_b; p.gate_a = gate_a; p.gate_b = gate_b; p.cap = cap;
  p.gates = reinterpret_cast<float4*>(gates); p.norm_state = norm_state; p.norm_dim = norm_dim; p.tokens = tokens;
  B200_REQUIRE(aligned16(gates), B200_E_ALIGN, "memory_prepare: gates must be 16-byte aligned");
  return dtype == B200F_BF16 ? launch_prepare(p, (bf16*)out, batch, (cudaStream_t)s) : launch_prepare(p, (float*)out, batch, (cudaStream_t)s);
}

extern "C" size_t b200f_memory_scan_ws_bytes(int64_t tokens, int batch, int max_q, int heads, int dim, int vdim, int kind, int dtype) {
  if (kind != B200F_MEMORY_DELTA || !chunks_fit(dtype, dim, vdim, max_q)) return 0;
  return (size_t)(tokens / kChunk + batch + 1) * heads * 2 * kChunk * kChunk * sizeof(bf16);
}

extern "C" int b200f_memory_scan(const void* rows, int dtype, int64_t row_pitch, int64_t q_off, int64_t k_off, int64_t v_off,
                                 int qk_heads, int heads, int dim, int vdim, int kind, float* gates, float q_scale,
                                 const float* skip, float* state, float* norm_state, const int32_t* slots,
                                 const int32_t* positions, const int32_t* seq_start, float* out, float* den, int64_t tokens,
                                 int batch, int max_q, void* ws, int simple, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype) && valid_kind(kind), B200_E_UNSUPPORTED, "memory_scan: dtype %d, kind %d", dtype, kind);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && batch >= 0 && batch < 65536 && heads > 0 && heads < 65536 && qk_heads > 0 &&
                   heads % qk_heads == 0 && dim > 0 && vdim > 0 && max_q > 0 && (seq_start || tokens == batch),
               B200_E_SHAPE, "memory_scan: tokens=%lld batch=%d heads=%d/%d dim=%d vdim=%d", (long long)tokens, batch, heads, qk_heads, dim, vdim);
  B200_REQUIRE(dim <= 512, B200_E_UNSUPPORTED, "memory_scan: dim %d is above 512", dim);
  const int64_t hq = (dim + 7) & ~7, vp = (vdim + 7) & ~7;
  B200_REQUIRE(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + qk_heads * hq <= row_pitch && k_off + qk_heads * hq <= row_pitch &&
                   v_off + heads * vp <= row_pitch, B200_E_SHAPE, "memory_scan: heads do not fit into rows of %lld", (long long)row_pitch);
  if (tokens == 0 || batch == 0) return B200_OK;
  B200_REQUIRE(rows && gates && state && slots && positions && out && (kind != B200F_MEMORY_EXP || (norm_state && den)), B200_E_NULL, "memory_scan: null pointer");
  B200_REQUIRE(aligned16(rows) && aligned16(gates) && aligned16(state) && row_pitch % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0,
               B200_E_ALIGN, "memory_scan: rows and heads must start on 16-byte boundaries");
  MemoryParams p{row_pitch, q_off, k_off, v_off, qk_heads, heads, dim, vdim, reinterpret_cast<float4*>(gates), q_scale, skip, state, norm_state,
                 slots, positions, seq_start, out, den, 0};
  if (seq_start && !simple && chunks_fit(dtype, dim, vdim, max_q)) {
    B200_REQUIRE(kind != B200F_MEMORY_DELTA || (ws && aligned16(ws)), B200_E_NULL, "memory_scan: no workspace");
    const bf16* r = (const bf16*)rows;
    switch (kind) {
      case B200F_MEMORY_EXP: return launch_chunks<B200F_MEMORY_EXP>(p, r, nullptr, tokens, batch, max_q, (cudaStream_t)s);
      case B200F_MEMORY_SSD: return launch_chunks<B200F_MEMORY_SSD>(p, r, nullptr, tokens, batch, max_q, (cudaStream_t)s);
      default: return launch_chunks<B200F_MEMORY_DELTA>(p, r, (bf16*)ws, tokens, batch, max_q, (cudaStream_t)s);
    }
  }
  return dtype == B200F_BF16 ? launch_memory(p, kind, (const bf16*)rows, batch, (cudaStream_t)s)
                             : launch_memory(p, kind, (const float*)rows, batch, (cudaStream_t)s);
}

extern "C" int b200f_memory_scan_status(int* out_host, int reset) {
  B200_REQUIRE(out_host, B200_E_NULL, "memory_scan_status: null pointer");
  cudaError_t e = cudaMemcpyFromSymbol(out_host, g_gemm_status, sizeof(int));
  if (e == cudaSuccess && reset) {
    const int zero = 0;
    e = cudaMemcpyToSymbol(g_gemm_status, &zero, sizeof(int));
  }
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "memory_scan_status: %s", cudaGetErrorString(e));
  return B200_OK;
}

extern "C" int b200f_memory_output(const float* o, const float* den, int heads, int vdim, int group, const float* y, int splits,
                                   int64_t split_stride, int64_t y_pitch, int64_t gate_col, int gate, const float* norm_w,
                                   int norm_len, float eps, void* out, int64_t out_pitch, int dtype, int64_t tokens,
                                   b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype) && gate >= B200F_GATE_SILU_BEFORE && gate <= B200F_GATE_SILU_AFTER, B200_E_UNSUPPORTED,
               "memory_output: dtype %d, gate %d", dtype, gate);
  const int64_t n = (int64_t)heads * vdim;
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && heads > 0 && vdim > 0 && group > 0 && n % group == 0 && norm_len > 0 && n % norm_len == 0 &&
                   splits >= 1 && gate_col >= 0 && gate_col + n <= y_pitch && out_pitch >= n, B200_E_SHAPE,
               "memory_output: tokens=%lld heads=%d vdim=%d group=%d", (long long)tokens, heads, vdim, group);
  B200_REQUIRE((norm_len == n || norm_len == group) && (!den || group == vdim), B200_E_UNSUPPORTED,
               "memory_output: gains of %d for groups of %d, divisors per head of %d", norm_len, group, vdim);
  if (tokens == 0) return B200_OK;
  B200_REQUIRE(o && y && norm_w && out, B200_E_NULL, "memory_output: null pointer");
  MemoryOutput p{o, den, heads, vdim, group, y, splits, split_stride, y_pitch, gate_col, gate, norm_w, norm_len, eps, out_pitch, tokens, 1, 1};
  const int64_t groups = n / group;
  const bool by4 = group % 4 == 0 && y_pitch % 4 == 0 && gate_col % 4 == 0 && split_stride % 4 == 0 && out_pitch % 4 == 0 && aligned16(o) && aligned16(y) &&
                   aligned16(norm_w) && aligned16(out);
  const int v = by4 && (group >= 128 || group % 2) ? 4 : (by4 && group >= 32 ? 2 : 1);      // narrow packs keep the lanes busy in small groups
  if (groups < 8 && group > 32 * v * kOutKeep) p.wpg = (int)(8 / groups);
  else
    while (p.cta_rows < 8 && (2 * p.cta_rows * n <= 4096 || p.cta_rows * groups < 8) && tokens >= 16ll * p.cta_rows * sm_count()) p.cta_rows *= 2;
  const dim3 grid((unsigned)((tokens + p.cta_rows - 1) / p.cta_rows)), block(256);
  cudaStream_t st = (cudaStream_t)s;
  if (dtype == B200F_BF16) {
    if (v == 4) launch_pdl(memory_output_kernel<bf16, 4>, grid, block, 0, st, p, (bf16*)out);
    else if (v == 2) launch_pdl(memory_output_kernel<bf16, 2>, grid, block, 0, st, p, (bf16*)out);
    else launch_pdl(memory_output_kernel<bf16, 1>, grid, block, 0, st, p, (bf16*)out);
  } else {
    if (v == 4) launch_pdl(memory_output_kernel<float, 4>, grid, block, 0, st, p, (float*)out);
    else if (v == 2) launch_pdl(memory_output_kernel<float, 2>, grid, block, 0, st, p, (float*)out);
    else launch_pdl(memory_output_kernel<float, 1>, grid, block, 0, st, p, (float*)out);
  }
  return check_launch("memory_output");
}
