// GGUF block types known to the device code (plain C++: host bindings include it too).
#pragma once

namespace oxb {

// GGUF tensor type codes (subset with device decoders)
enum QuantType : int {
  kQ_F32 = 0,
  kQ_F16 = 1,
  kQ_Q4_0 = 2,
  kQ_Q4_1 = 3,
  kQ_Q5_0 = 6,
  kQ_Q5_1 = 7,
  kQ_Q8_0 = 8,
  kQ_Q2_K = 10,
  kQ_Q3_K = 11,
  kQ_Q4_K = 12,
  kQ_Q5_K = 13,
  kQ_Q6_K = 14,
  kQ_IQ4_NL = 20,
  kQ_BF16 = 30,
  kQ_TQ2_0 = 35,
  kQ_NVFP4 = 144,
};

// Block types with an integer (dp4a) GEMV and an in-kernel expansion in the GEMM.
inline bool mmvq_has_int8_path(int qtype) {
  switch (qtype) {
    case kQ_Q4_0: case kQ_Q4_1: case kQ_Q5_0: case kQ_Q5_1: case kQ_Q8_0: case kQ_Q4_K: case kQ_Q5_K: case kQ_Q6_K:
      return true;
    default:
      return false;
  }
}

// Bytes of one packed row of K values, -1 for a type without a device decoder.
inline long long quant_row_bytes(int qtype, long long K) {
  switch (qtype) {
    case kQ_F32: return K * 4;
    case kQ_F16: case kQ_BF16: return K * 2;
    case kQ_Q4_0: case kQ_IQ4_NL: return K / 32 * 18;
    case kQ_Q4_1: return K / 32 * 20;
    case kQ_Q5_0: return K / 32 * 22;
    case kQ_Q5_1: return K / 32 * 24;
    case kQ_Q8_0: return K / 32 * 34;
    case kQ_Q2_K: return K / 256 * 84;
    case kQ_Q3_K: return K / 256 * 110;
    case kQ_Q4_K: return K / 256 * 144;
    case kQ_Q5_K: return K / 256 * 176;
    case kQ_Q6_K: return K / 256 * 210;
    case kQ_TQ2_0: return K / 256 * 66;
    case kQ_NVFP4: return K / 16 * 16;
    default: return -1;
  }
}

}  // namespace oxb
