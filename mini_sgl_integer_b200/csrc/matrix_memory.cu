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
// memory_scan_kernel      prompts: a CTA per (sequence, head, slice of columns) keeps its part of S in registers over all
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

// (first, second) gate of one token and head, as the scan reads them: EXP log gates (f, i), SSD (decay, dt), DELTA (decay, beta).
__device__ __forceinline__ float2 memory_gates(const MemoryPrepare& p, const float* row, int h) {
  const float a = part_sum(row + p.gate_col_a + h, p.splits, p.split_stride);
  if (p.kind == B200F_MEMORY_EXP) {
    const float b = part_sum(row + p.gate_col_b + h, p.splits, p.split_stride);
    const float f = p.cap * tanhf((a + p.gate_a[h]) / p.cap), i = p.cap * tanhf((b + p.gate_b[h]) / p.cap);
    return make_float2(-softplus_f32(-f), i);
  }
  const float dt = softplus_f32(a + p.gate_b[h]);
  const float decay = expf(-expf(p.gate_a[h]) * dt);
  if (p.kind == B200F_MEMORY_SSD) return make_float2(decay, dt);
  return make_float2(decay, sigmoid_f32(part_sum(row + p.gate_col_b + h, p.splits, p.split_stride)));
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
        r = make_float4(expf(fm - m), expf(g.y - m), expf(-m), 0.0f);
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
  const float4* gates;
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
        if (lane == 0) *reinterpret_cast<float4*>(sc + 4 * t) = make_float4(rg[t].x, rg[t].y, 1.0f / sqrtf(sk + kUnitEps), p.q_scale / sqrtf(sq + kUnitEps));
      } else if (lane == 0) {
        *reinterpret_cast<float4*>(sc + 4 * t) = make_float4(rg[t].x, rg[t].y, rg[t].z, p.q_scale);
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

// Log gates (f, i) of a prompt batch to (exp(f + m_(t-1) - m_t), exp(i - m_t), exp(-m_t)); a warp per (sequence, head).
__global__ void __launch_bounds__(32)
running_max_kernel(const MemoryPrepare p) {
  __shared__ float2 fi[32];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, seq = blockIdx.y, lane = threadIdx.x;
  const int64_t t0 = p.seq_start[seq], t1 = p.seq_start[seq + 1];
  if (t0 >= t1) return;
  float* ms = p.norm_state + ((int64_t)p.slots[seq] * p.heads + h) * (p.norm_dim + 1) + p.norm_dim;
  float m = p.positions[t0] > 0 ? *ms : 0.0f;
  float4 next = t0 + lane < t1 ? p.gates[(t0 + lane) * p.heads + h] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  for (int64_t base = t0; base < t1; base += 32) {
    const int n = (int)min((int64_t)32, t1 - base);
    const float4 g = next;
    __syncwarp();
    fi[lane] = make_float2(g.x, g.y);
    __syncwarp();
    if (base + 32 + lane < t1) next = p.gates[(base + 32 + lane) * p.heads + h];
    float before = m, after = m;
    for (int t = 0; t < n; ++t) {
      const float2 u = fi[t];
      const float nm = fmaxf(u.x + m, u.y);
      if (t == lane) { before = m; after = nm; }
      m = nm;
    }
    if (lane < n) p.gates[(base + lane) * p.heads + h] = make_float4(expf(g.x + before - after), expf(g.y - after), expf(-after), 0.0f);
  }
  if (lane == 0) *ms = m;
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
};

template <typename T>
__global__ void __launch_bounds__(256)
memory_output_kernel(const MemoryOutput p, T* __restrict__ out) {
  extern __shared__ __align__(16) unsigned char smem[];
  float* u = reinterpret_cast<float*>(smem);          // [heads * vdim]
  __shared__ float part[8];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int n = p.heads * p.vdim, groups = n / p.group;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* o = p.o + row * n;
  const float* gate = p.y + row * p.y_pitch + p.gate_col;
  const int wpg = groups >= 8 ? 1 : 8 / groups, at_once = 8 / wpg, sub = warp % wpg;       // warps per group
  for (int g0 = 0; g0 < groups; g0 += at_once) {
    const int g = g0 + warp / wpg;
    const bool live = warp / wpg < at_once && g < groups;
    float ss = 0.0f;
    if (live) {
      for (int i = sub * 32 + lane; i < p.group; i += 32 * wpg) {
        const int c = g * p.group + i;
        float v = o[c];
        if (p.den) v /= p.den[row * p.heads + c / p.vdim];
        if (p.gate == B200F_GATE_SILU_BEFORE) v *= silu_f32(part_sum(gate + c, p.splits, p.split_stride));
        u[c] = v;
        ss = fmaf(v, v, ss);
      }
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
    const float inv = 1.0f / sqrtf(ss / (float)p.group + p.eps);
    for (int i = sub * 32 + lane; i < p.group; i += 32 * wpg) {
      const int c = g * p.group + i;
      float v = u[c] * inv * p.norm_w[c % p.norm_len];
      if (p.gate != B200F_GATE_SILU_BEFORE) {
        const float z = part_sum(gate + c, p.splits, p.split_stride);
        v *= p.gate == B200F_GATE_SIGMOID_AFTER ? sigmoid_f32(z) : silu_f32(z);
      }
      out[row * p.out_pitch + c] = from_f32<T>(v);
    }
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

extern "C" int b200f_memory_scan(const void* rows, int dtype, int64_t row_pitch, int64_t q_off, int64_t k_off, int64_t v_off,
                                 int qk_heads, int heads, int dim, int vdim, int kind, const float* gates, float q_scale,
                                 const float* skip, float* state, float* norm_state, const int32_t* slots,
                                 const int32_t* positions, const int32_t* seq_start, float* out, float* den, int64_t tokens,
                                 int batch, b200_stream_t s) {
  B200_REQUIRE(valid_dtype(dtype) && valid_kind(kind), B200_E_UNSUPPORTED, "memory_scan: dtype %d, kind %d", dtype, kind);
  B200_REQUIRE(tokens >= 0 && tokens < (1ll << 31) && batch >= 0 && batch < 65536 && heads > 0 && heads < 65536 && qk_heads > 0 &&
                   heads % qk_heads == 0 && dim > 0 && vdim > 0 && (seq_start || tokens == batch),
               B200_E_SHAPE, "memory_scan: tokens=%lld batch=%d heads=%d/%d dim=%d vdim=%d", (long long)tokens, batch, heads, qk_heads, dim, vdim);
  B200_REQUIRE(dim <= 512, B200_E_UNSUPPORTED, "memory_scan: dim %d is above 512", dim);
  const int64_t hq = (dim + 7) & ~7, vp = (vdim + 7) & ~7;
  B200_REQUIRE(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + qk_heads * hq <= row_pitch && k_off + qk_heads * hq <= row_pitch &&
                   v_off + heads * vp <= row_pitch, B200_E_SHAPE, "memory_scan: heads do not fit into rows of %lld", (long long)row_pitch);
  if (tokens == 0 || batch == 0) return B200_OK;
  B200_REQUIRE(rows && gates && state && slots && positions && out && (kind != B200F_MEMORY_EXP || (norm_state && den)), B200_E_NULL, "memory_scan: null pointer");
  B200_REQUIRE(aligned16(rows) && aligned16(gates) && aligned16(state) && row_pitch % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0,
               B200_E_ALIGN, "memory_scan: rows and heads must start on 16-byte boundaries");
  MemoryParams p{row_pitch, q_off, k_off, v_off, qk_heads, heads, dim, vdim, reinterpret_cast<const float4*>(gates), q_scale, skip, state, norm_state,
                 slots, positions, seq_start, out, den, 0};
  return dtype == B200F_BF16 ? launch_memory(p, kind, (const bf16*)rows, batch, (cudaStream_t)s)
                             : launch_memory(p, kind, (const float*)rows, batch, (cudaStream_t)s);
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
  B200_REQUIRE(n * 4 <= 200 * 1024, B200_E_UNSUPPORTED, "memory_output: rows of %lld values are too wide", (long long)n);
  if (tokens == 0) return B200_OK;
  B200_REQUIRE(o && y && norm_w && out, B200_E_NULL, "memory_output: null pointer");
  MemoryOutput p{o, den, heads, vdim, group, y, splits, split_stride, y_pitch, gate_col, gate, norm_w, norm_len, eps, out_pitch};
  const size_t bytes = (size_t)n * 4;
  cudaError_t e = dtype == B200F_BF16 ? cudaFuncSetAttribute(memory_output_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes)
                                      : cudaFuncSetAttribute(memory_output_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
  B200_REQUIRE(e == cudaSuccess, B200_E_CUDA, "memory_output: cudaFuncSetAttribute: %s", cudaGetErrorString(e));
  if (dtype == B200F_BF16) launch_pdl(memory_output_kernel<bf16>, dim3((unsigned)tokens), dim3(256), bytes, (cudaStream_t)s, p, (bf16*)out);
  else launch_pdl(memory_output_kernel<float>, dim3((unsigned)tokens), dim3(256), bytes, (cudaStream_t)s, p, (float*)out);
  return check_launch("memory_output");
}
