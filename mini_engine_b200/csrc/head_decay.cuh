// What the kernels of head_decay.cu (any sizes, on the CUDA cores) and head_decay_mma.cu (prompts of bfloat16, on the tensor cores) share:
// the arguments, and a token's factor and decay.  See head_decay.cu for the recurrence.
#pragma once
#include "common.cuh"

constexpr int HD_LC = 64, HD_VT = 64;
constexpr double HD_LOG2E = 1.4426950408889634074;

struct HdArgs {
  const void *q, *k, *v;
  int64_t ldq, ldk, ldv;
  int H, G, D, V;
  float k_scale;
  const float* dt;            // null: the constant form
  int64_t ld_dt;
  const float *dt_bias, *a_log, *decay;
  const double* log2_decay;
  const float* skip;
  float* S;
  const int *cu, *ctx, *slots;
  float* o;
};

// The factor g of token row t, head h, and the natural logarithm of its decay (the state-space form).
__device__ __forceinline__ void hd_step_size(const HdArgs& a, int64_t t, int h, float& gain, float& log_a) {
  const float z = a.dt[t * a.ld_dt + h] + a.dt_bias[h];
  gain = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
  log_a = -expf(a.a_log[h]) * gain;
}
// The factor g and log2 of the decay; the factor g and the decay itself.
__device__ __forceinline__ void hd_token_log2(const HdArgs& a, int64_t t, int h, float& gain, double& log2_a) {
  gain = a.k_scale;
  if (a.dt) {
    float log_a;
    hd_step_size(a, t, h, gain, log_a);
    log2_a = (double)log_a * HD_LOG2E;
  } else {
    log2_a = a.log2_decay[h];
  }
}
__device__ __forceinline__ void hd_token(const HdArgs& a, int64_t t, int h, float& gain, float& decay) {
  gain = a.k_scale;
  if (a.dt) {
    float log_a;
    hd_step_size(a, t, h, gain, log_a);
    decay = expf(log_a);
  } else {
    decay = a.decay[h];
  }
}

// A run's numbers for one head: the inclusive sums B of log2 a and the factors g, zero factors and no further decay beyond its tokens.  The
// kernel that makes the runs' states leaves them in global memory for the two behind it.
struct HdRun {
  double b[HD_LC];
  float g[HD_LC];
};

// The first warp's work.
__device__ __forceinline__ void hd_run_scalars(const HdArgs& a, int tok0, int L, int h, float* g_s, double* b_s) {
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x, t0 = 2 * lane, t1 = t0 + 1;
  float g0 = 0.f, g1 = 0.f;
  double l0 = 0.0, l1 = 0.0;
  if (t0 < L) hd_token_log2(a, tok0 + t0, h, g0, l0);
  if (t1 < L) hd_token_log2(a, tok0 + t1, h, g1, l1);
  const double pair = l0 + l1;
  double run = pair;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double up = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += up;
  }
  g_s[t0] = g0;
  g_s[t1] = g1;
  b_s[t0] = run - pair + l0;
  b_s[t1] = run;
}
