// The residual stream takes what is pending and is normed (RMS), one pass:
//
//   x <- x + sum_i f_i(y_i) + va + vb          up to three outputs y_i [T, W] of the block before and two vectors of W values
//   f(y) = s * y                               s: a weight of W values (a layer scale), or none
//   f(y) = s * y / sqrt(mean(y^2) + eps_y)     an output that passes an RMS norm of its own before it joins
//   out = x / sqrt(mean(x^2) + eps) * w        (``w`` null: out = x, a copy of the stream in the output's type)
//
// Rows of ``out`` may lie further apart than W (a copy beside other columns).  The residual stream, sums, statistics and weights are
// float32 and a row's sums are taken in a fixed order.  With ``rows`` only those rows are read and x is left as it is (the model's
// last norm at the places whose logits are wanted).
#include "common.cuh"

struct StreamTerm {
  const void* y;
  const float* scale;       // [W] or null
  float eps;                // of the output's own norm; negative: none
};
struct StreamArgs {
  float* x;
  StreamTerm t[3];
  int n_terms;
  const float *va, *vb, *w;
  int64_t out_ld;
  float eps;
  const int* rows;
  int W;
};

__device__ __forceinline__ void sn_load4(const float* p, float (&v)[4]) {
  const float4 t = *reinterpret_cast<const float4*>(p);
  v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
__device__ __forceinline__ void sn_load4(const bf16* p, float (&v)[4]) {
  const uint2 t = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&t.x), b = *reinterpret_cast<const __nv_bfloat162*>(&t.y);
  v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
}
__device__ __forceinline__ void sn_store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void sn_store4(bf16* p, const float (&v)[4]) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
}

// Three block sums at once, in a fixed order.
__device__ __forceinline__ void sn_block_sum3(float (&s)[3], float (*red)[32]) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int i = 0; i < 3; ++i) s[i] = warp_sum(s[i]);
  __syncthreads();
  if (lane == 0)
#pragma unroll
    for (int i = 0; i < 3; ++i) red[i][warp] = s[i];
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    float total = 0.f;
    for (int w = 0; w < nwarps; ++w) total += red[i][w];
    s[i] = total;
  }
}

// A row a block, in registers: four neighbours a thread and turn, PER turns.  W is a multiple of four, pointers and row lengths allow
// 16-byte accesses (8-byte for bfloat16).
template <typename TY, typename TO, int PER>
__global__ void __launch_bounds__(1024) stream_norm_kernel(StreamArgs a, TO* __restrict__ out) {
  __shared__ float red3[3][32], red[32];
  const int W = a.W;
  pdl_wait();
  pdl_launch_dependents();
  const int64_t r = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  float* xr = a.x + r * W;
  float v[PER][4], y[3][PER][4];
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = 4 * (threadIdx.x + p * blockDim.x);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[p][j] = y[0][p][j] = y[1][p][j] = y[2][p][j] = 0.f;
    if (i >= W) continue;
    sn_load4(xr + i, v[p]);
#pragma unroll
    for (int k = 0; k < 3; ++k)
      if (k < a.n_terms) sn_load4(reinterpret_cast<const TY*>(a.t[k].y) + r * W + i, y[k][p]);
  }
  float f[3] = {1.f, 1.f, 1.f};
  if (a.t[0].eps >= 0.f || a.t[1].eps >= 0.f || a.t[2].eps >= 0.f) {          // (the same in all threads; absent terms have a negative eps)
    float s[3] = {0.f, 0.f, 0.f};
#pragma unroll
    for (int p = 0; p < PER; ++p)
#pragma unroll
      for (int k = 0; k < 3; ++k)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[k] = fmaf(y[k][p][j], y[k][p][j], s[k]);
    sn_block_sum3(s, red3);
#pragma unroll
    for (int k = 0; k < 3; ++k)
      if (a.t[k].eps >= 0.f) f[k] = 1.0f / sqrtf(s[k] / (float)W + a.t[k].eps);
  }
  const bool changed = a.n_terms > 0 || a.va || a.vb;
  float ss = 0.f;
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = 4 * (threadIdx.x + p * blockDim.x);
    if (i >= W) continue;
    float t[4];
#pragma unroll
    for (int k = 0; k < 3; ++k) {
      if (k >= a.n_terms) continue;
      if (a.t[k].scale) {
        sn_load4(a.t[k].scale + i, t);
#pragma unroll
        for (int j = 0; j < 4; ++j) v[p][j] = fmaf(y[k][p][j] * f[k], t[j], v[p][j]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) v[p][j] = fmaf(y[k][p][j], f[k], v[p][j]);
      }
    }
    if (a.va) { sn_load4(a.va + i, t); for (int j = 0; j < 4; ++j) v[p][j] += t[j]; }
    if (a.vb) { sn_load4(a.vb + i, t); for (int j = 0; j < 4; ++j) v[p][j] += t[j]; }
    if (changed && !a.rows) sn_store4(xr + i, v[p]);
#pragma unroll
    for (int j = 0; j < 4; ++j) ss = fmaf(v[p][j], v[p][j], ss);
  }
  const float rs = a.w ? 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps) : 1.f;
  TO* o = out + (int64_t)blockIdx.x * a.out_ld;
#pragma unroll
  for (int p = 0; p < PER; ++p) {
    const int i = 4 * (threadIdx.x + p * blockDim.x);
    if (i >= W) continue;
    if (a.w) {
      float t[4];
      sn_load4(a.w + i, t);
#pragma unroll
      for (int j = 0; j < 4; ++j) v[p][j] = v[p][j] * rs * t[j];
    }
    sn_store4(o + i, v[p]);
  }
}

// The same for any W, one value a thread and turn; the row's new values wait in shared memory.
template <typename TY, typename TO>
__global__ void __launch_bounds__(256) stream_norm_any_kernel(StreamArgs a, TO* __restrict__ out) {
  extern __shared__ float row[];
  __shared__ float red3[3][32], red[32];
  const int W = a.W;
  pdl_wait();
  pdl_launch_dependents();
  const int64_t r = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  float* xr = a.x + r * W;
  float f[3] = {1.f, 1.f, 1.f}, s[3] = {0.f, 0.f, 0.f};
  for (int i = threadIdx.x; i < W; i += blockDim.x)
#pragma unroll
    for (int k = 0; k < 3; ++k)
      if (k < a.n_terms && a.t[k].eps >= 0.f) {
        const float y = to_f<TY>(reinterpret_cast<const TY*>(a.t[k].y)[r * W + i]);
        s[k] = fmaf(y, y, s[k]);
      }
  sn_block_sum3(s, red3);
#pragma unroll
  for (int k = 0; k < 3; ++k)
    if (k < a.n_terms && a.t[k].eps >= 0.f) f[k] = 1.0f / sqrtf(s[k] / (float)W + a.t[k].eps);
  const bool changed = a.n_terms > 0 || a.va || a.vb;
  float ss = 0.f;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    float v = xr[i];
#pragma unroll
    for (int k = 0; k < 3; ++k)
      if (k < a.n_terms) v = fmaf(to_f<TY>(reinterpret_cast<const TY*>(a.t[k].y)[r * W + i]) * f[k], a.t[k].scale ? a.t[k].scale[i] : 1.f, v);
    if (a.va) v += a.va[i];
    if (a.vb) v += a.vb[i];
    if (changed && !a.rows) xr[i] = v;
    row[i] = v;
    ss = fmaf(v, v, ss);
  }
  const float rs = a.w ? 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps) : 1.f;
  TO* o = out + (int64_t)blockIdx.x * a.out_ld;
  for (int i = threadIdx.x; i < W; i += blockDim.x) o[i] = from_f<TO>(a.w ? row[i] * rs * a.w[i] : row[i]);      // (what the thread wrote itself)
}

// x: [T, W] float32.  y0, y1, y2: [T, W] of y_dtype or null (the ones in front of a null are there); scale0.. : [W] float32 or null;
// eps0..: of the output's own norm, negative for none.  va, vb, w: [W] float32 or null.  out: [n, W] of out_dtype, rows out_ld
// elements apart.  rows: [n] int32 or null (then n == T).
ME_API int me_stream_norm(float* x, const void* y0, const void* y1, const void* y2, int y_dtype, const float* scale0, const float* scale1,
                          const float* scale2, float eps0, float eps1, float eps2, const float* va, const float* vb, const float* w,
                          float eps, void* out, int out_dtype, int64_t out_ld, const int* rows, int n, int W, cudaStream_t stream) {
  if (n == 0) return 0;
  ME_REQUIRE(n > 0 && W > 0 && W <= 49152 && out_ld >= W, "me_stream_norm: bad sizes n=%d W=%d out_ld=%lld", n, W, (long long)out_ld);
  ME_REQUIRE(!(y1 && !y0) && !(y2 && !y1), "me_stream_norm: outputs are given in order");
  const StreamArgs a = {x, {{y0, scale0, y0 ? eps0 : -1.f}, {y1, scale1, y1 ? eps1 : -1.f}, {y2, scale2, y2 ? eps2 : -1.f}},
                        y2 ? 3 : (y1 ? 2 : (y0 ? 1 : 0)), va, vb, w, out_ld, eps, rows, W};
  auto off = [](const void* p, size_t to) { return p && ((uintptr_t)p % to) != 0; };
  const size_t y_al = y_dtype == ME_F32 ? 16 : 8, o_al = out_dtype == ME_F32 ? 16 : 8;
  const bool vec = W % 4 == 0 && W <= 16384 && out_ld % 4 == 0 && !off(x, 16) && !off(y0, y_al) && !off(y1, y_al) && !off(y2, y_al) && !off(scale0, 16) &&
                   !off(scale1, 16) && !off(scale2, 16) && !off(va, 16) && !off(vb, 16) && !off(w, 16) && !off(out, o_al);
  // (which kernel and how many threads follow from W and the pointers alone, so a row's sums are the same in every batch)
  if (vec) {
    const int quads = W / 4, per = quads <= 256 ? 1 : (quads <= 2048 ? 2 : 4);
    const int threads = ((quads + per - 1) / per + 31) / 32 * 32;
#define SN_PER(PER_) \
  if (per == PER_) me_launch(stream_norm_kernel<TY, TO, PER_>, dim3(n), dim3(threads), 0, stream, a, (TO*)out)
    ME_DISPATCH_DTYPE(y_dtype, TY, ME_DISPATCH_DTYPE(out_dtype, TO, { SN_PER(1); SN_PER(2); SN_PER(4); }));
#undef SN_PER
  } else {
    const size_t smem = sizeof(float) * W;
    ME_DISPATCH_DTYPE(y_dtype, TY, ME_DISPATCH_DTYPE(out_dtype, TO, {
      if (smem > 40 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(stream_norm_any_kernel<TY, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        ME_REQUIRE(e == cudaSuccess, "me_stream_norm: cannot raise shared memory: %s", cudaGetErrorString(e));
      }
      me_launch(stream_norm_any_kernel<TY, TO>, dim3(n), dim3(W >= 256 ? 256 : (W >= 128 ? 128 : 64)), smem, stream, a, (TO*)out);
    }));
  }
  ME_LAUNCH_CHECK("me_stream_norm");
  return 0;
}
