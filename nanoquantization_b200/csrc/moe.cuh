// Shared by the mixture-of-experts kernels.
#pragma once
#include "mixers.cuh"
#include "nqb200_moe.h"

namespace nqb200 {

struct MoeArgs {
  const void* x; const void* w; void* out;
  int kind, tokens, N, K, experts, top;
  nqb200_moe_plan plan;
  int dtype, out_dtype;
  int* status;
  cudaStream_t stream;
};

constexpr int kMoeDecodeTokens = 16;   // up to here every expert's weights are streamed once by the decode kernel

bool moe_decode_supports(int64_t tokens, int64_t N, int64_t K);
int moe_decode(const MoeArgs& a);
bool moe_umma_supports(int64_t tokens, int64_t N, int64_t K, int64_t top);
int moe_umma(const MoeArgs& a);

}  // namespace nqb200
