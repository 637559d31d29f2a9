// RMS norm in groups, on the output of a sub-layer rather than on its input:
//
//   a row of W values is cut into ``groups`` equal consecutive parts; every part is divided by its own
//   sqrt(mean(part^2) + eps) and the whole row is multiplied by a weight of W values.
//
// Three uses, one kernel (a row a block, statistics and the stream in float32):
//   add     residual[t] += norm(y[t]) * w        a sub-layer's output joins the stream normalised (the sub-layers read
//                                                the stream itself); ``copy`` [T, W] receives the new stream in the
//                                                working dtype for the products of the next sub-layer
//   self    residual[t] <- norm(residual[t]) * w the norm behind the embedding, with the same copy
//   rows    out[i] = norm(residual[rows[i]]) * w the model's last norm at the wanted places; the stream is left alone
#include "common.cuh"

// Four neighbouring values of a row at a time where the row allows it (W a multiple of 4 and 16-byte aligned rows), so that a
// thread has all its loads in flight at once; else one value at a time.
template <typename T, bool VEC>
__device__ __forceinline__ void load4(const T* __restrict__ p, float (&f)[4]) {
  if (VEC) {
    if constexpr (sizeof(T) == 4) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      f[0] = q.x; f[1] = q.y; f[2] = q.z; f[3] = q.w;
    } else {
      const uint2 q = *reinterpret_cast<const uint2*>(p);
      const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&q.x), b = *reinterpret_cast<const __nv_bfloat162*>(&q.y);
      f[0] = __low2float(a); f[1] = __high2float(a); f[2] = __low2float(b); f[3] = __high2float(b);
    }
  } else {
    f[0] = to_f<T>(p[0]);
  }
}

template <typename T, bool VEC>
__device__ __forceinline__ void store4(T* __restrict__ p, const float (&f)[4]) {
  if (VEC) {
    if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
      const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
      uint2 q;
      q.x = *reinterpret_cast<const uint32_t*>(&a);
      q.y = *reinterpret_cast<const uint32_t*>(&b);
      *reinterpret_cast<uint2*>(p) = q;
    }
  } else {
    p[0] = from_f<T>(f[0]);
  }
}

template <typename TY, typename TO, bool VEC>
__global__ void __launch_bounds__(256)
group_norm_kernel(float* __restrict__ residual, const TY* __restrict__ y, int64_t y_stride, const float* __restrict__ w,
                  int groups, float eps, TO* __restrict__ out, const int* __restrict__ rows, int W) {
  extern __shared__ __align__(16) float vals[];   // [W] the row that is normalised, then [groups] its factors
  pdl_wait();
  pdl_launch_dependents();
  constexpr int V = VEC ? 4 : 1;
  float* factor = vals + W;
  const int i = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
  const int64_t t = rows ? rows[i] : i;
  float* res = residual + t * W;
  for (int d = tid * V; d < W; d += blockDim.x * V) {
    float f[4];
    if (y) load4<TY, VEC>(y + t * y_stride + d, f);
    else load4<float, VEC>(res + d, f);
#pragma unroll
    for (int k = 0; k < V; ++k) vals[d + k] = f[k];
  }
  __syncthreads();
  const int n = W / groups;
  for (int g = warp; g < groups; g += warps) {
    float ss = 0.f;
    for (int d = lane; d < n; d += 32) ss = fmaf(vals[g * n + d], vals[g * n + d], ss);
    ss = warp_sum(ss);
    if (lane == 0) factor[g] = 1.0f / sqrtf(ss / (float)n + eps);
  }
  __syncthreads();
  for (int d = tid * V; d < W; d += blockDim.x * V) {
    float wv[4], rv[4], o[4];
    load4<float, VEC>(w + d, wv);
    const bool adds = rows == nullptr && y != nullptr;
    if (adds) load4<float, VEC>(res + d, rv);
#pragma unroll
    for (int k = 0; k < V; ++k) o[k] = vals[d + k] * factor[(d + k) / n] * wv[k] + (adds ? rv[k] : 0.f);
    if (rows == nullptr) store4<float, VEC>(res + d, o);
    if (out) store4<TO, VEC>(out + (int64_t)i * W + d, o);
  }
}

// residual: [T, W] float32.  y: [T, >= W] rows of ``y_dtype`` or null (the stream itself is normalised).  w: [W] float32.
// out: [n, W] of ``out_dtype`` or null.  rows: [n] int32 or null (then n = T and the stream is renewed).
ME_API int me_group_norm(float* residual, const void* y, int y_dtype, int64_t y_stride, const float* w, int groups, float eps,
                         void* out, int out_dtype, const int* rows, int n, int W, cudaStream_t stream) {
  if (n == 0) return 0;
  ME_REQUIRE(n > 0 && W > 0 && groups >= 1 && W % groups == 0, "me_group_norm: %d values do not split into %d groups", W, groups);
  ME_REQUIRE(!(rows && y), "me_group_norm: the wanted rows are normalised from the stream, not from an output");
  ME_REQUIRE(!rows || out, "me_group_norm: the wanted rows need a place to go");
  const size_t smem = sizeof(float) * ((size_t)W + groups);
  ME_REQUIRE(smem <= 200 * 1024, "me_group_norm: rows of %d values are too long", W);
  const int y_size = y ? (y_dtype == ME_BF16 ? 2 : 4) : 4, out_size = out ? (out_dtype == ME_BF16 ? 2 : 4) : 4;
  const bool vec = W % 4 == 0 && ((uintptr_t)residual & 15) == 0 && ((uintptr_t)w & 15) == 0 &&
                   (!y || (((uintptr_t)y) % (4 * y_size) == 0 && (y_stride * y_size) % (4 * y_size) == 0)) &&
                   (!out || ((uintptr_t)out) % (4 * out_size) == 0);
  const dim3 block(W >= 4096 ? 256 : 128);
  ME_DISPATCH_DTYPE(y ? y_dtype : ME_F32, TY, ME_DISPATCH_DTYPE(out ? out_dtype : ME_F32, TO, {
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(group_norm_kernel<TY, TO, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (e == cudaSuccess) e = cudaFuncSetAttribute(group_norm_kernel<TY, TO, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      ME_REQUIRE(e == cudaSuccess, "me_group_norm: cannot raise shared memory: %s", cudaGetErrorString(e));
    }
    if (vec)
      me_launch(group_norm_kernel<TY, TO, true>, dim3(n), block, smem, stream, residual, (const TY*)y, y_stride, w, groups, eps, (TO*)out,
                rows, W);
    else
      me_launch(group_norm_kernel<TY, TO, false>, dim3(n), block, smem, stream, residual, (const TY*)y, y_stride, w, groups, eps,
                (TO*)out, rows, W);
  }));
  ME_LAUNCH_CHECK("me_group_norm");
  return 0;
}

// The norm behind a recurrence: a row of y is cut into ``groups`` equal parts, each divided by its own sqrt(mean^2 + eps), with the gate
// silu(z) in front of the norm or behind it and an optional weight:
//   first:  u = y silu(z),  out = u / rms_g(u) * w          else:  out = y / rms_g(y) * w * silu(z)
// LANES threads a (row, group) pair: a warp for short groups (several pairs a block), a block for long ones; values are read twice (the
// second time from the cache close by).
template <typename TZ, typename TO, int LANES, bool VEC>
__global__ void __launch_bounds__(256)
gated_group_norm_kernel(const float* __restrict__ y, int64_t y_ld, const TZ* __restrict__ z, int64_t z_ld, const float* __restrict__ w, int gate_first,
                        float eps, TO* __restrict__ out, int64_t out_ld, int64_t pairs, int groups, int n) {
  __shared__ float red[32];
  constexpr int V = VEC ? 4 : 1;
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x % LANES;
  const int64_t pair = (int64_t)blockIdx.x * (blockDim.x / LANES) + threadIdx.x / LANES;
  if (LANES == 32 && pair >= pairs) return;
  const int64_t t = pair / groups;
  const int c0 = (int)(pair - t * groups) * n;
  const float* yr = y + t * y_ld + c0;
  const TZ* zr = z + t * z_ld + c0;
  auto gated = [&](int i, float (&u)[4], float (&s)[4]) {      // u: what is normed; s: silu(z)
    load4<float, VEC>(yr + i, u);
    load4<TZ, VEC>(zr + i, s);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      s[j] = s[j] / (1.f + expf(-s[j]));
      if (gate_first) u[j] *= s[j];
    }
  };
  float ss = 0.f;
  for (int i = lane * V; i < n; i += LANES * V) {
    float u[4], s[4];
    if (gate_first) gated(i, u, s);
    else load4<float, VEC>(yr + i, u);
#pragma unroll
    for (int j = 0; j < V; ++j) ss = fmaf(u[j], u[j], ss);
  }
  ss = LANES == 32 ? warp_sum(ss) : block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / (float)n + eps);
  for (int i = lane * V; i < n; i += LANES * V) {
    float u[4], s[4], f[4];
    gated(i, u, s);
    if (w) load4<float, VEC>(w + c0 + i, f);
#pragma unroll
    for (int j = 0; j < V; ++j) u[j] = u[j] * r * (w ? f[j] : 1.f) * (gate_first ? 1.f : s[j]);
    store4<TO, VEC>(out + t * out_ld + c0 + i, u);
  }
}

// y: [T, W] float32 rows; z: [T, W] of z_dtype; w: [W] float32 or null; out: [T, W] of out_dtype.  Rows lie *_ld elements apart.
ME_API int me_gated_group_norm(const float* y, int64_t y_ld, const void* z, int z_dtype, int64_t z_ld, const float* w, int gate_first, float eps,
                               void* out, int out_dtype, int64_t out_ld, int T, int W, int groups, cudaStream_t stream) {
  if (T == 0) return 0;
  ME_REQUIRE(T > 0 && W > 0 && groups > 0 && W % groups == 0, "me_gated_group_norm: %d groups of %d values", groups, W);
  const int n = W / groups;
  auto off = [](const void* p, size_t to) { return p && ((uintptr_t)p % to) != 0; };
  const bool vec = n % 4 == 0 && y_ld % 4 == 0 && z_ld % 4 == 0 && out_ld % 4 == 0 && !off(y, 16) && !off(z, z_dtype == ME_F32 ? 16 : 8) && !off(w, 16) &&
                   !off(out, out_dtype == ME_F32 ? 16 : 8);
  const bool warps = n <= (vec ? 512 : 128);
  const int64_t pairs = (int64_t)T * groups;
  const int threads = warps ? (pairs >= 4096 ? 256 : 64) : 256;
  const int64_t blocks = warps ? (pairs + threads / 32 - 1) / (threads / 32) : pairs;
  ME_REQUIRE(blocks < (1ll << 31), "me_gated_group_norm: too many rows");
#define GGN_CASE(LANES_, VEC_)                                                                                                              \
  me_launch(gated_group_norm_kernel<TZ, TO, LANES_, VEC_>, dim3((unsigned)blocks), dim3(threads), 0, stream, y, y_ld, (const TZ*)z, z_ld, w, \
            gate_first, eps, (TO*)out, out_ld, pairs, groups, n)
  ME_DISPATCH_DTYPE(z_dtype, TZ, ME_DISPATCH_DTYPE(out_dtype, TO, {
    if (warps) { if (vec) GGN_CASE(32, true); else GGN_CASE(32, false); }
    else { if (vec) GGN_CASE(256, true); else GGN_CASE(256, false); }
  }));
#undef GGN_CASE
  ME_LAUNCH_CHECK("me_gated_group_norm");
  return 0;
}
