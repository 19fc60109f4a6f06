// Per-step bookkeeping of a decode batch on the device (positions, KV locations, lengths); part of every library.
#include "common.cuh"

namespace b200 {

// ---------------------------------------------------------------------------------------------------
// One decode step of bookkeeping for `batch` sequences, all on the device so that the step can be
// replayed from a CUDA graph: the new token of sequence b sits at position seq_lens[b]; its KV slot
// is page_table[b][pos / 16] * 16 + pos % 16; the sequence then has pos + 1 keys.
// ---------------------------------------------------------------------------------------------------
__global__ void decode_prepare_kernel(const int32_t* __restrict__ page_table, int64_t pitch, int32_t* __restrict__ seq_lens,
                                      int32_t* __restrict__ positions, int32_t* __restrict__ out_loc,
                                      int32_t* __restrict__ kv_lens, int batch, int max_len) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= batch) return;
  int pos = seq_lens[b];
  pos = pos < 0 ? 0 : (pos > max_len - 1 ? max_len - 1 : pos);      // a full sequence rewrites its last slot
  const int page = page_table[(int64_t)b * pitch + (pos >> 4)];
  positions[b] = pos;
  out_loc[b] = page * 16 + (pos & 15);
  kv_lens[b] = pos + 1;
  seq_lens[b] = pos + 1;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_decode_prepare(const int32_t* page_table, int64_t table_pitch, int32_t* seq_lens, int32_t* positions,
                                   int32_t* out_loc, int32_t* kv_lens, int batch, int max_len, b200_stream_t s) {
  B200_REQUIRE(batch >= 0 && max_len > 0 && table_pitch >= (max_len + 15) / 16, B200_E_SHAPE,
               "decode_prepare: batch=%d max_len=%d table_pitch=%lld", batch, max_len, (long long)table_pitch);
  if (batch == 0) return B200_OK;
  B200_REQUIRE(page_table && seq_lens && positions && out_loc && kv_lens, B200_E_NULL, "decode_prepare: null pointer");
  launch_pdl(decode_prepare_kernel, dim3((batch + 127) / 128), dim3(128), 0, (cudaStream_t)s, page_table, table_pitch, seq_lens, positions, out_loc,
             kv_lens, batch, max_len);
  return check_launch("decode_prepare");
}
