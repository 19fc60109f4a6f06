// Library-wide pieces of the integer path's C ABI: version, compiled-in tables.
#include <cstring>

#include "common.cuh"
#include "luts.inc"

namespace b200 {

static const int32_t h_inv_sqrt_lut[1024] = {B200_LUT_kInvSqrtLut};
static const int32_t h_exp2_silu_lut[1024] = {B200_LUT_kExp2SiluLut};
static const int32_t h_exp2_attn_lut[1024] = {B200_LUT_kExp2AttnLut};

}  // namespace b200

extern "C" int b200_version(void) { return 100; }

extern "C" int b200_get_lut(int which, int32_t* out_host_1024) {
  B200_REQUIRE(out_host_1024, B200_E_NULL, "get_lut: null pointer");
  const int32_t* src = which == 0   ? b200::h_inv_sqrt_lut
                       : which == 1 ? b200::h_exp2_silu_lut
                       : which == 2 ? b200::h_exp2_attn_lut
                                    : nullptr;
  B200_REQUIRE(src, B200_E_SHAPE, "get_lut: which=%d (0, 1 or 2)", which);
  memcpy(out_host_1024, src, 1024 * sizeof(int32_t));
  return B200_OK;
}
