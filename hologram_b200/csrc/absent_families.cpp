// Stands in for the kernel families a serving build leaves out (LUT activations, the reference-exact matmul and decode
// attention, quantized products, tensor parallelism): a call that needs one is refused.
#include "common.h"

namespace {
int32_t absent(const char* what) {
    return holo_fail(HOLO_ERR_UNSUPPORTED_OP, "unsupported op: this is a serving build without the %s kernels (run hologram_b200/build.py for all of them)", what);
}
}  // namespace

int32_t holo_lut_table(holo_b200_ctx*, uint8_t, uint8_t, const uint16_t**) { return absent("LUT activation"); }
int32_t holo_launch_lut(holo_b200_ctx*, const uint16_t*, const uint16_t*, uint16_t*, uint64_t) { return absent("LUT activation"); }
int32_t holo_launch_decode_attention(holo_b200_ctx*, const HoloAttnArgs&) { return absent("decode attention"); }
int32_t holo_launch_matmul(holo_b200_ctx*, const void*, const void*, void*, uint32_t, uint32_t, uint32_t, uint8_t, uint8_t, const void*, bool) { return absent("matmul"); }
int32_t holo_launch_matmul_add_activation(holo_b200_ctx*, const void*, const void*, void*, uint32_t, uint32_t, uint32_t, uint8_t, uint8_t, const void*) { return absent("matmul"); }
int32_t holo_launch_matmul_multi(holo_b200_ctx*, const void*, const void*, uint32_t, uint32_t, uint32_t, uint8_t, const HoloMatmulSeg*, uint32_t) { return absent("matmul"); }
bool holo_matmul_head_ops_ok(uint32_t, uint32_t, uint32_t, uint8_t, const HoloMatmulSeg*, uint32_t) { return false; }
int32_t holo_launch_matmul_dequant_kn(holo_b200_ctx*, const float*, const uint8_t*, const float*, const int32_t*, const float*, float*, uint32_t, uint32_t, uint32_t,
                                      uint32_t, uint32_t, uint8_t, float, int32_t, int) { return absent("quantized product"); }
int32_t holo_launch_matmul_e8cb_omajor(holo_b200_ctx*, const float*, const uint8_t*, const int8_t*, const float*, const int32_t*, const float*, float*, uint32_t,
                                       uint32_t, uint32_t, int) { return absent("quantized product"); }
int32_t holo_launch_matmul_w8a8_omajor(holo_b200_ctx*, const float*, const int8_t*, const float*, const int32_t*, const float*, float*, uint32_t, uint32_t, uint32_t,
                                       int, bool) { return absent("quantized product"); }
int32_t holo_all_reduce(holo_b200_ctx*, void*, uint64_t, uint8_t) { return absent("tensor-parallel"); }
int32_t holo_all_reduce_add(holo_b200_ctx*, const void*, const void*, void*, uint64_t, uint8_t) { return absent("tensor-parallel"); }
void holo_tp_destroy(holo_b200_ctx*) {}

extern "C" {
int32_t holo_b200_decode_attention_q8_static(void*, const void*, const int8_t*, const float*, const int8_t*, const float*, const int8_t*, const float*, const int8_t*,
                                             const float*, const uint32_t*, void*, uint32_t, uint32_t, uint32_t, uint32_t, uint32_t, uint32_t, uint8_t) {
    return absent("decode attention");
}
int32_t holo_b200_decode_attention_q8_static_status(void*) { return absent("decode attention"); }
int32_t holo_b200_nccl_unique_id(uint8_t*) { return absent("tensor-parallel"); }
int32_t holo_b200_ctx_init_tp(holo_b200_ctx*, const uint8_t*, int32_t, int32_t) { return absent("tensor-parallel"); }
int32_t holo_b200_ctx_init_tp_timeout(holo_b200_ctx*, const uint8_t*, int32_t, int32_t, uint32_t) { return absent("tensor-parallel"); }
int32_t holo_b200_ctx_tp_transport(holo_b200_ctx*) { return 0; }
int32_t holo_b200_tp_emulate_all_reduce(holo_b200_ctx*, int32_t, const void* const*, const void* const*, void* const*, uint64_t, uint8_t, int32_t) {
    return absent("tensor-parallel");
}
int32_t holo_b200_tp_emulate_all_reduce_ex(holo_b200_ctx*, int32_t, const void* const*, const void* const*, void* const*, uint64_t, uint8_t, int32_t, int32_t, uint32_t) {
    return absent("tensor-parallel");
}
}
