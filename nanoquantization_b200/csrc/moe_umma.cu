#include "moe.cuh"
namespace nqb200 {
bool moe_umma_supports(int64_t, int64_t, int64_t, int64_t) { return false; }
int moe_umma(const MoeArgs&) { return NQB200_ERR_BAD_SHAPE; }
}
