/* nqb200_moe -- C ABI of the mixture-of-experts kernels (sm_100a): routing of tokens to experts, and the experts' linears
 * over tokens grouped by expert.
 *
 * Conventions as in nqb200_mixers.h: plain device pointers, asynchronous on `stream`, status codes, nothing here allocates.
 * A pair (t, k) is a token and one of the `top` experts it was sent to; its number is t * top + k. */
#ifndef NQB200_MOE_H
#define NQB200_MOE_H

#include "nqb200.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef struct {
  int32_t experts, top;
  int32_t groups, keep;       /* experts form `groups` equal runs of neighbours; only the `keep` best can be chosen from */
  float scale;
  const float* correction;    /* [experts], added to the scores for the choice only; or NULL */
} nqb200_router;

/* What routing leaves: pairs sorted by expert. */
typedef struct {
  int32_t* expert;            /* [tokens * top] expert of each pair */
  float* weight;              /* [tokens * top] */
  int32_t* offsets;           /* [experts + 1]: expert e has order[offsets[e]] .. order[offsets[e + 1] - 1] */
  int32_t* order;             /* [tokens * top] pair numbers */
  int32_t* active;            /* [experts + 1]: how many experts have tokens, then which */
  int32_t* counters;          /* [2 * experts] scratch */
} nqb200_moe_plan;

/* s = sigmoid(logits) (float [tokens, experts]), choice = s + correction.  A group's score is the sum of its two largest
 * choices; in the `keep` best groups the `top` largest choices are taken, weight = s / (sum of the chosen s + 1e-20) *
 * scale.  Ties go to the lower index. */
int nqb200_moe_route(const float* logits, const nqb200_router* r, const nqb200_moe_plan* plan, int64_t tokens, void* stream);

/* One linear of all experts, w [experts, N, K] of dtype, over the plan's pairs.  With i counting pairs in the plan's order:
 *   up    x [tokens, K], row order[i] / top;  out [tokens * top, N] of dtype, row i = gelu(w x), exact (erf)
 *   down  x [tokens * top, K], row i;         out [tokens * top, N] of out_dtype, row order[i] = weight * (w x) */
enum { NQB200_MOE_UP = 0, NQB200_MOE_DOWN = 1 };
int nqb200_moe_linear(const void* x, const void* w, void* out, int kind, int64_t tokens, int64_t N, int64_t K,
                      const nqb200_router* r, const nqb200_moe_plan* plan, int dtype, int out_dtype, int* status, void* stream);
/* The kernel that a call takes: "decode", "tcgen05" or "simple". */
const char* nqb200_moe_linear_kernel(int64_t tokens, int64_t N, int64_t K, int64_t top, int dtype);

#ifdef __cplusplus
}
#endif
#endif
