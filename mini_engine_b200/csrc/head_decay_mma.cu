// The prompt kernels of head_decay.cu on the tensor cores (mma.sync m16n8k16, bfloat16 in, float32 accumulate), for bfloat16 q, k and v.
//
// q, k and v enter the products as they are.  What is float32 (the state, the weighted scores, the weighted values) enters as the
// sum of three bfloat16 numbers, x = hi + mid + lo, each the rounding of what the ones before left: 24 digits, float32's own.  A
// product of such a factor with a bfloat16 one is three products added in float32, so the results are those of float32 products
// up to the order of sums.
//
//   hd_mma_state_kernel   U = k^T (g_s 2^(B_L - B_s) v_s) of a run: 64 tokens x 64 columns a block, a warp a strip of 16 rows by 32 columns
//   hd_mma_out_kernel     a warp takes 16 tokens of the run and 32 columns: q S_in (three parts), scaled by 2^(B_t); then, 16 keys at a time up to the
//                         diagonal, the scores q k^T, their weights in the registers, and the product with v (three parts)
#include "head_decay.cuh"
#include "mma_prims.cuh"

namespace {

using namespace mma_prims;

constexpr int HM_SR = 64;                     // rows of the state that hd_mma_out_kernel holds in shared memory at a time
constexpr int HM_LDV = HD_VT + 8;             // bfloat16 elements of a row of 64 columns in shared memory (an odd number of 16-byte pieces)

// Two floats as a pair of bfloat16 (x in the lower half) in each of the three parts.
__device__ __forceinline__ void split3_pair(float x, float y, uint32_t (&p)[3]) {
  p[0] = pack_bf16(x, y);
  x -= __uint_as_float(p[0] << 16);
  y -= __uint_as_float(p[0] & 0xffff0000u);
  p[1] = pack_bf16(x, y);
  p[2] = pack_bf16(x - __uint_as_float(p[1] << 16), y - __uint_as_float(p[1] & 0xffff0000u));
}

// HD_LC rows of cols (a multiple of 8) bfloat16 values into shared memory by asynchronous copies of a block of 256, zeros beyond n_rows and
// n_cols.  Eight neighbouring threads take a row's pieces of 16 bytes.
__device__ __forceinline__ void hm_fill(bf16* dst, int ld_dst, int cols, const bf16* src, int64_t ld_src, int n_rows, int n_cols) {
  const int r0 = threadIdx.x >> 3, c0 = (threadIdx.x & 7) * 8;
#pragma unroll
  for (int i = 0; i < HD_LC / 32; ++i) {
    const int r = r0 + 32 * i;
    const bf16* s = src + (int64_t)r * ld_src;
    for (int c = c0; c < cols; c += 64) {
      const bool ok = r < n_rows && c < n_cols;
      cp_async16(dst + r * ld_dst + c, ok ? s + c : src, ok);
    }
  }
}

// One block = one run x one head x HD_VT columns of U; nums[c, h]: the run's numbers.
__global__ void __launch_bounds__(256)
hd_mma_state_kernel(HdArgs a, const int* __restrict__ tiles, float* __restrict__ states, HdRun* __restrict__ nums) {
  extern __shared__ __align__(16) unsigned char hm_smem[];
  __shared__ float g_s[HD_LC];
  __shared__ double b_s[HD_LC];
  constexpr int LC = HD_LC, VT = HD_VT, LDV = HM_LDV;
  const int D = a.D, V = a.V, D16 = (D + 15) / 16 * 16, ldk = D16 + 8;
  bf16* Ks = reinterpret_cast<bf16*>(hm_smem);  // [LC][ldk]
  bf16* Ws = Ks + LC * ldk;                     // [3][LC][LDV]: g_s 2^(B_L - B_s) v_s in three parts
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, v0 = blockIdx.z * VT;
  const int b = tiles[2 * blockIdx.x], q0 = tiles[2 * blockIdx.x + 1];
  const int tok0 = a.cu[b] + q0, L = min(LC, a.cu[b + 1] - tok0);
  pdl_wait();
  pdl_launch_dependents();
  if (L <= 0) return;
  const int g = h / (a.H / a.G);
  hm_fill(Ks, ldk, D16, reinterpret_cast<const bf16*>(a.k) + (int64_t)tok0 * a.ldk + (int64_t)g * D, a.ldk, L, D);
  cp_async_commit();
  // this thread's 16 values (two rows' pieces of eight columns), on their way while the first warp sums the decays
  const bf16* vsrc = reinterpret_cast<const bf16*>(a.v) + (int64_t)tok0 * a.ldv + (int64_t)h * V + v0;
  uint4 raw[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = tid / 8 + 32 * i, c = tid % 8 * 8;
    raw[i] = r < L && v0 + c < V ? *reinterpret_cast<const uint4*>(vsrc + (int64_t)r * a.ldv + c) : make_uint4(0, 0, 0, 0);
  }
  hd_run_scalars(a, tok0, L, h, g_s, b_s);
  __syncthreads();
  const double bl = b_s[LC - 1];
  if (tid < LC && blockIdx.z == 0) {
    HdRun& run = nums[(int64_t)blockIdx.x * a.H + h];
    run.b[tid] = b_s[tid];
    run.g[tid] = g_s[tid];
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = tid / 8 + 32 * i, c = tid % 8 * 8;
    const float f = g_s[r] * exp2f((float)(bl - b_s[r]));
    const __nv_bfloat162* x = reinterpret_cast<const __nv_bfloat162*>(&raw[i]);
    uint32_t p[4][3];
#pragma unroll
    for (int j = 0; j < 4; ++j) split3_pair(__low2float(x[j]) * f, __high2float(x[j]) * f, p[j]);
#pragma unroll
    for (int k = 0; k < 3; ++k) *reinterpret_cast<uint4*>(Ws + (k * LC + r) * LDV + c) = make_uint4(p[0][k], p[1][k], p[2][k], p[3][k]);
  }
  cp_async_wait<0>();
  __syncthreads();
  const int mr = lane & 7, mj = lane >> 3;
  float* out = states + ((int64_t)blockIdx.x * a.H + h) * D * V;
  for (int u = warp; u < D16 / 8; u += 8) {     // strips of 16 rows (key channels) x 32 columns
    const int d0 = u / 2 * 16, c0 = u % 2 * 32;
    if (v0 + c0 >= V) continue;
    float acc[4][4] = {};
#pragma unroll
    for (int ks = 0; ks < LC / 16; ++ks) {
      if (16 * ks >= L) break;                  // (zeros from here on)
      uint32_t ka[4];
      ldmatrix_x4_trans(ka, Ks + (16 * ks + mr + (mj >= 2 ? 8 : 0)) * ldk + d0 + (mj & 1 ? 8 : 0));
#pragma unroll
      for (int p = 0; p < 3; ++p)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          uint32_t vb[4];
          ldmatrix_x4_trans(vb, Ws + (p * LC + 16 * ks + mr + (mj & 1 ? 8 : 0)) * LDV + c0 + 16 * n + (mj >= 2 ? 8 : 0));
          mma_bf16(acc[2 * n], ka, vb[0], vb[1]);
          mma_bf16(acc[2 * n + 1], ka, vb[2], vb[3]);
        }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int c = v0 + c0 + 8 * n + 2 * (lane & 3), d = d0 + (lane >> 2);
      if (c >= V) continue;
      if (d < D) *reinterpret_cast<float2*>(out + (int64_t)d * V + c) = make_float2(acc[n][0], acc[n][1]);
      if (d + 8 < D) *reinterpret_cast<float2*>(out + (int64_t)(d + 8) * V + c) = make_float2(acc[n][2], acc[n][3]);
    }
  }
}

// One block = one run x one head x HD_VT columns; states[c] holds the state in front of the run.
__global__ void __launch_bounds__(256, 3)
hd_mma_out_kernel(HdArgs a, const int* __restrict__ tiles, const float* __restrict__ states, const HdRun* __restrict__ nums) {
  extern __shared__ __align__(16) unsigned char hm_smem[];
  __shared__ float g_s[HD_LC];
  __shared__ double b_s[HD_LC];
  constexpr int LC = HD_LC, VT = HD_VT, LDV = HM_LDV;
  const int D = a.D, V = a.V, D16 = (D + 15) / 16 * 16, ldk = D16 + 8;
  bf16* Qs = reinterpret_cast<bf16*>(hm_smem);  // [LC][ldk]
  bf16* Ks = Qs + LC * ldk;                     // [LC][ldk]
  bf16* Vs = Ks + LC * ldk;                     // [LC][LDV]
  bf16* Ss = Vs + LC * LDV;                     // [3][HM_SR][LDV]: rows of the state in three parts
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, v0 = blockIdx.z * VT;
  const int b = tiles[2 * blockIdx.x], q0 = tiles[2 * blockIdx.x + 1];
  const int tok0 = a.cu[b] + q0, L = min(LC, a.cu[b + 1] - tok0);
  pdl_wait();
  pdl_launch_dependents();
  if (L <= 0) return;
  const int g = h / (a.H / a.G);
  hm_fill(Qs, ldk, D16, reinterpret_cast<const bf16*>(a.q) + (int64_t)tok0 * a.ldq + (int64_t)g * D, a.ldq, L, D);
  hm_fill(Ks, ldk, D16, reinterpret_cast<const bf16*>(a.k) + (int64_t)tok0 * a.ldk + (int64_t)g * D, a.ldk, L, D);
  hm_fill(Vs, LDV, VT, reinterpret_cast<const bf16*>(a.v) + (int64_t)tok0 * a.ldv + (int64_t)h * V + v0, a.ldv, L, V - v0);
  cp_async_commit();
  // HM_SR rows of the state at a time: into registers (on their way while the products of the rows before run), then split into shared memory
  const int sr = tid / 16, scol = tid % 16 * 4;
  const float* ssrc = states + ((int64_t)blockIdx.x * a.H + h) * D * V + v0 + scol;
  float4 sx[HM_SR / 16];
  auto fetch_rows = [&](int d0) {
#pragma unroll
    for (int i = 0; i < HM_SR / 16; ++i) {
      const int d = d0 + sr + 16 * i;
      sx[i] = d < D && v0 + scol < V ? *reinterpret_cast<const float4*>(ssrc + (int64_t)d * V) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  auto store_rows = [&]() {
#pragma unroll
    for (int i = 0; i < HM_SR / 16; ++i) {
      uint32_t p0[3], p1[3];
      split3_pair(sx[i].x, sx[i].y, p0);
      split3_pair(sx[i].z, sx[i].w, p1);
#pragma unroll
      for (int k = 0; k < 3; ++k) *reinterpret_cast<uint2*>(Ss + (k * HM_SR + sr + 16 * i) * LDV + scol) = make_uint2(p0[k], p1[k]);
    }
  };
  fetch_rows(0);
  if (tid < LC) {
    const HdRun& run = nums[(int64_t)blockIdx.x * a.H + h];
    b_s[tid] = run.b[tid];
    g_s[tid] = run.g[tid];
  }
  store_rows();
  cp_async_wait<0>();
  __syncthreads();
  const int r0 = 16 * (warp >> 1), c0 = 32 * (warp & 1);
  const bool active = r0 < L && v0 + c0 < V;
  const int mr = lane & 7, mj = lane >> 3, t0 = r0 + (lane >> 2), t1 = t0 + 8;
  float acc[4][4] = {};
  const bf16* q_at = Qs + (r0 + mr + (mj & 1 ? 8 : 0)) * ldk + (mj >= 2 ? 8 : 0);
  const bf16* s_at = Ss + (mr + (mj & 1 ? 8 : 0)) * LDV + c0 + (mj >= 2 ? 8 : 0);
  for (int s0 = 0; s0 < D16; s0 += HM_SR) {
    const bool more = s0 + HM_SR < D16;
    if (more) fetch_rows(s0 + HM_SR);
    if (active) {
#pragma unroll
      for (int j = 0; j < HM_SR / 16; ++j) {
        if (s0 + 16 * j >= D16) break;
        uint32_t qa[4];
        ldmatrix_x4(qa, q_at + s0 + 16 * j);
#pragma unroll
        for (int p = 0; p < 3; ++p)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            uint32_t sb[4];
            ldmatrix_x4_trans(sb, s_at + (p * HM_SR + 16 * j) * LDV + 16 * n);
            mma_bf16(acc[2 * n], qa, sb[0], sb[1]);
            mma_bf16(acc[2 * n + 1], qa, sb[2], sb[3]);
          }
      }
    }
    if (more) {                                 // (the same in all threads)
      __syncthreads();
      store_rows();
      __syncthreads();
    }
  }
  if (!active) return;
  const double bt0 = b_s[t0], bt1 = b_s[t1];
  {
    const float f0 = exp2f((float)bt0), f1 = exp2f((float)bt1);
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      acc[n][0] *= f0; acc[n][1] *= f0;
      acc[n][2] *= f1; acc[n][3] *= f1;
    }
  }
  // Weights of keys in front of the diagonal block: 2^(B_t - B_s) = 2^(B_t - r) 2^(r - B_s) with r the sum up to the last token in front of
  // this warp's; both exponents are <= 0.  On the diagonal every (query, key) has an exponential of its own.
  const double ref = r0 > 0 ? b_s[r0 - 1] : 0.0;
  const float e0 = exp2f((float)(bt0 - ref)), e1 = exp2f((float)(bt1 - ref));
  for (int s0 = 0; s0 <= r0; s0 += 16) {        // keys up to the diagonal
    float sc[2][4] = {};
    const bf16* k_at = Ks + (s0 + mr + (mj >= 2 ? 8 : 0)) * ldk + (mj & 1 ? 8 : 0);
    for (int d0 = 0; d0 < D16; d0 += 16) {
      uint32_t qa[4], kb[4];
      ldmatrix_x4(qa, q_at + d0);
      ldmatrix_x4(kb, k_at + d0);
      mma_bf16(sc[0], qa, kb[0], kb[1]);
      mma_bf16(sc[1], qa, kb[2], kb[3]);
    }
    uint32_t pa[3][4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int s = s0 + 8 * n + 2 * (lane & 3);
      const double bs0 = b_s[s], bs1 = b_s[s + 1];
      const float g0 = g_s[s], g1 = g_s[s + 1];
      float w0, w1, w2, w3;
      if (s0 < r0) {
        const float f0 = g0 * exp2f((float)(ref - bs0)), f1 = g1 * exp2f((float)(ref - bs1));
        w0 = sc[n][0] * (e0 * f0); w1 = sc[n][1] * (e0 * f1);
        w2 = sc[n][2] * (e1 * f0); w3 = sc[n][3] * (e1 * f1);
      } else {
        w0 = s <= t0 ? sc[n][0] * g0 * exp2f((float)(bt0 - bs0)) : 0.f; w1 = s + 1 <= t0 ? sc[n][1] * g1 * exp2f((float)(bt0 - bs1)) : 0.f;
        w2 = s <= t1 ? sc[n][2] * g0 * exp2f((float)(bt1 - bs0)) : 0.f; w3 = s + 1 <= t1 ? sc[n][3] * g1 * exp2f((float)(bt1 - bs1)) : 0.f;
      }
      uint32_t lo[3], hi[3];
      split3_pair(w0, w1, lo);
      split3_pair(w2, w3, hi);
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        pa[p][2 * n] = lo[p];
        pa[p][2 * n + 1] = hi[p];
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      uint32_t vb[4];
      ldmatrix_x4_trans(vb, Vs + (s0 + mr + (mj & 1 ? 8 : 0)) * LDV + c0 + 16 * n + (mj >= 2 ? 8 : 0));
#pragma unroll
      for (int p = 0; p < 3; ++p) {
        mma_bf16(acc[2 * n], pa[p], vb[0], vb[1]);
        mma_bf16(acc[2 * n + 1], pa[p], vb[2], vb[3]);
      }
    }
  }
  const float skip = a.skip ? a.skip[h] : 0.f;
  float* o0 = a.o + (int64_t)(tok0 + t0) * a.H * V + (int64_t)h * V + v0;
  float* o1 = o0 + (int64_t)8 * a.H * V;
#pragma unroll
  for (int n = 0; n < 4; ++n) {
    const int c = c0 + 8 * n + 2 * (lane & 3);
    if (v0 + c >= V) continue;
    if (a.skip) {
      const __nv_bfloat162 x0 = *reinterpret_cast<const __nv_bfloat162*>(Vs + t0 * LDV + c), x1 = *reinterpret_cast<const __nv_bfloat162*>(Vs + t1 * LDV + c);
      acc[n][0] = fmaf(skip, __low2float(x0), acc[n][0]);
      acc[n][1] = fmaf(skip, __high2float(x0), acc[n][1]);
      acc[n][2] = fmaf(skip, __low2float(x1), acc[n][2]);
      acc[n][3] = fmaf(skip, __high2float(x1), acc[n][3]);
    }
    if (t0 < L) *reinterpret_cast<float2*>(o0 + c) = make_float2(acc[n][0], acc[n][1]);
    if (t1 < L) *reinterpret_cast<float2*>(o1 + c) = make_float2(acc[n][2], acc[n][3]);
  }
}

size_t state_smem(int D) { return sizeof(bf16) * ((size_t)HD_LC * ((D + 15) / 16 * 16 + 8) + 3 * HD_LC * HM_LDV); }
size_t out_smem(int D) {
  const size_t D16 = (D + 15) / 16 * 16;
  return sizeof(bf16) * (2 * HD_LC * (D16 + 8) + HD_LC * HM_LDV + 3 * HM_SR * HM_LDV);
}

}  // namespace

// bfloat16 rows that start on 16 bytes, sizes in whole pieces of eight.
bool me_head_decay_mma_takes(const HdArgs& a, int dtype) {
  auto ok = [](const void* p, int64_t ld) { return ((uintptr_t)p % 16) == 0 && ld % 8 == 0; };
  return dtype == ME_BF16 && a.D % 8 == 0 && a.V % 8 == 0 && a.D <= 256 && ok(a.q, a.ldq) && ok(a.k, a.ldk) && ok(a.v, a.ldv) &&
         ((uintptr_t)a.o % 16) == 0 && out_smem(a.D) <= 220 * 1024;
}

int me_head_decay_mma_states(const HdArgs& a, const int* tiles, int n_tiles, float* states, HdRun* nums, cudaStream_t stream) {
  const size_t smem = state_smem(a.D);
  cudaError_t e = cudaFuncSetAttribute(hd_mma_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  ME_REQUIRE(e == cudaSuccess, "me_head_decay_scan: cannot raise shared memory to %zu: %s", smem, cudaGetErrorString(e));
  me_launch(hd_mma_state_kernel, dim3(n_tiles, a.H, (a.V + HD_VT - 1) / HD_VT), dim3(256), smem, stream, a, tiles, states, nums);
  return 0;
}

int me_head_decay_mma_out(const HdArgs& a, const int* tiles, int n_tiles, const float* states, const HdRun* nums, cudaStream_t stream) {
  const size_t smem = out_smem(a.D);
  cudaError_t e = cudaFuncSetAttribute(hd_mma_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  ME_REQUIRE(e == cudaSuccess, "me_head_decay_scan: cannot raise shared memory to %zu: %s", smem, cudaGetErrorString(e));
  me_launch(hd_mma_out_kernel, dim3(n_tiles, a.H, (a.V + HD_VT - 1) / HD_VT), dim3(256), smem, stream, a, tiles, states, nums);
  return 0;
}
