// The difference of two attention maps: head h of the output takes the results a_0, a_1 of query heads 2h and 2h + 1 (the
// same values weighed by two softmaxes), o = a_0 - lambda a_1, divided by its root mean square over the head's V values
// (sqrt(mean(o^2) + eps), no weight) and times ``gain``.  float32 between the loads and the store; one warp a head of a token.
#include "common.cuh"

constexpr int DIFF_MAX = 256;

template <typename TI, typename TO>
__global__ void __launch_bounds__(128)
diff_combine_kernel(const TI* __restrict__ a, int64_t a_ld, TO* __restrict__ out, int64_t out_ld, int first, int n_tok, int H, int V, float lambda,
                    float gain, float eps) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t unit = (int64_t)blockIdx.x * 4 + warp;
  if (unit >= (int64_t)n_tok * H) return;
  const int t = first + (int)(unit / H), h = (int)(unit % H);
  const TI* a0 = a + (int64_t)t * a_ld + (int64_t)2 * h * V;
  float o[DIFF_MAX / 32], ss = 0.f;
#pragma unroll
  for (int i = 0; i < DIFF_MAX / 32; ++i) {
    const int d = lane + 32 * i;
    o[i] = d < V ? to_f<TI>(a0[d]) - lambda * to_f<TI>(a0[V + d]) : 0.f;
    ss = fmaf(o[i], o[i], ss);
  }
  const float r = gain / sqrtf(warp_sum(ss) / (float)V + eps);
  TO* dst = out + (int64_t)t * out_ld + (int64_t)h * V;
#pragma unroll
  for (int i = 0; i < DIFF_MAX / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < V) dst[d] = from_f<TO>(o[i] * r);
  }
}

// a: rows of 2*H*V values a_ld apart; out: rows of H*V values out_ld apart; rows [first, first + n_tok) of both.
ME_API int me_diff_combine(const void* a, int a_dtype, int64_t a_ld, void* out, int out_dtype, int64_t out_ld, int first, int n_tok, int H, int V,
                           float lambda, float gain, float eps, cudaStream_t stream) {
  if (n_tok == 0) return 0;
  ME_REQUIRE(n_tok > 0 && first >= 0 && H > 0 && V > 0 && V <= DIFF_MAX, "me_diff_combine: bad sizes T=%d H=%d V=%d", n_tok, H, V);
  const int64_t units = (int64_t)n_tok * H;
  ME_DISPATCH_DTYPE(a_dtype, TI, ME_DISPATCH_DTYPE(out_dtype, TO,
      me_launch(diff_combine_kernel<TI, TO>, dim3((unsigned)((units + 3) / 4)), dim3(128), 0, stream, (const TI*)a, a_ld, (TO*)out, out_ld, first,
                n_tok, H, V, lambda, gain, eps)));
  ME_LAUNCH_CHECK("me_diff_combine");
  return 0;
}
