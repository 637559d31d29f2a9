// A short causal convolution over time on each channel, with the last inputs of every request kept as state.
//
// out_t = [h_t +] sum_j w[:, j] * h_(t - taps + 1 + j), j = 0 .. taps-1, zeros before the request's first token.
// A request's portion of a step starts at position ``start`` = context length - tokens in the step; inputs at
// positions before ``start`` come from the request's state slot, which holds the last taps-1 inputs (state row k is
// position start - (taps-1) + k).  A second kernel then stores the last taps-1 inputs of the portion (moving old
// state rows up when the portion is shorter than taps-1).  A slot is never read for positions below 0, so a slot
// that another request used before needs no clearing.  Inputs, weights and state are float32.
#include "common.cuh"

template <typename TO>
__global__ void __launch_bounds__(256)
short_conv_kernel(const float* __restrict__ h, const float* __restrict__ wt, const float* __restrict__ state,
                  const int* __restrict__ token_req, const int* __restrict__ cu_seqlens,
                  const int* __restrict__ context_lens, const int* __restrict__ state_slots, TO* __restrict__ out,
                  int W, int taps, int add_input) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int w = blockIdx.y * blockDim.x + threadIdx.x;
  if (w >= W) return;
  const int b = token_req[t];
  const int tok0 = cu_seqlens[b], q_len = cu_seqlens[b + 1] - tok0;
  const int start = context_lens[b] - q_len;
  const int i = t - tok0;                         // local index in the portion
  const int slot = state_slots[b];
  float acc = add_input ? h[(int64_t)t * W + w] : 0.f;
  for (int j = 0; j < taps; ++j) {
    const int src = i - (taps - 1) + j;           // local index of the input
    if (start + src < 0) continue;                // before the request's first token
    float v;
    if (src >= 0) {
      v = h[(int64_t)(tok0 + src) * W + w];
    } else {
      if (slot < 0) continue;
      v = state[((int64_t)slot * (taps - 1) + (src + taps - 1)) * W + w];
    }
    acc = fmaf(wt[(int64_t)w * taps + j], v, acc);
  }
  out[(int64_t)t * W + w] = from_f<TO>(acc);
}

__global__ void __launch_bounds__(256)
short_conv_state_kernel(const float* __restrict__ h, float* __restrict__ state, const int* __restrict__ cu_seqlens,
                        const int* __restrict__ context_lens, const int* __restrict__ state_slots, int W, int taps) {
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.x;
  const int w = blockIdx.y * blockDim.x + threadIdx.x;
  if (w >= W) return;
  const int slot = state_slots[b];
  if (slot < 0) return;
  const int tok0 = cu_seqlens[b], n = cu_seqlens[b + 1] - tok0;
  if (n <= 0) return;
  const int start = context_lens[b] - n;
  float* st = state + (int64_t)slot * (taps - 1) * W + w;
  // Row k takes the input at local index n - (taps-1) + k.  Old rows are read at k + n > k, rows are written in
  // ascending order, so a thread never reads a row it has already replaced.
  for (int k = 0; k < taps - 1; ++k) {
    const int src = n - (taps - 1) + k;
    float v = 0.f;
    if (src >= 0) v = h[(int64_t)(tok0 + src) * W + w];
    else if (start + src >= 0) v = st[(int64_t)(src + taps - 1) * W];
    st[(int64_t)k * W] = v;
  }
}

// h: [T, W] float32.  wt: [W, taps] float32.  state: [slots, taps-1, W] float32 (unused when taps == 1).
// out: [T, W] of out_dtype.  update_state != 0 also runs the second kernel.
ME_API int me_short_conv(const float* h, const float* wt, float* state, const int* token_req, const int* cu_seqlens,
                         const int* context_lens, const int* state_slots, void* out, int out_dtype, int T, int B, int W,
                         int taps, int add_input, int update_state, cudaStream_t stream) {
  if (T == 0) return 0;
  ME_REQUIRE(T > 0 && B > 0 && W > 0 && taps >= 1, "me_short_conv: bad sizes T=%d B=%d W=%d taps=%d", T, B, W, taps);
  ME_REQUIRE(taps == 1 || state != nullptr, "me_short_conv: %d taps need a state", taps);
  const int threads = W >= 256 ? 256 : 64;
  dim3 grid(T, (W + threads - 1) / threads);
  ME_DISPATCH_DTYPE(out_dtype, TO,
                    me_launch(short_conv_kernel<TO>, grid, dim3(threads), 0, stream, h, wt, (const float*)state, token_req,
                              cu_seqlens, context_lens, state_slots, (TO*)out, W, taps, add_input));
  ME_LAUNCH_CHECK("me_short_conv");
  if (update_state && taps > 1) {
    me_launch(short_conv_state_kernel, dim3(B, (W + threads - 1) / threads), dim3(threads), 0, stream, h, state, cu_seqlens,
              context_lens, state_slots, W, taps);
    ME_LAUNCH_CHECK("me_short_conv (state)");
  }
  return 0;
}

// ---- the same on columns of a projection, with a bias and silu ---------------------------------------------------------------
//
// out_t = silu(b + sum_j w[:, j] * u_(t - taps + 1 + j)): u are C columns of float32 rows ld elements apart.  One block = up to CS_TILE tokens
// of one request x a strip of channels; a thread slides VEC channels' last inputs through registers, so that an input is read once (and
// taps - 1 times more at a tile's edge).  Requests that bring one token move their state on in this kernel; those that bring several
// leave it to conv_silu_state_kernel, since another block may still read the old rows.  TAPS 0: any number of taps, inputs read again.
constexpr int CS_TILE = 16;

template <int VEC> __device__ __forceinline__ void cs_load(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    v[0] = p[0];
  }
}
template <int VEC, typename TO> __device__ __forceinline__ void cs_store(TO* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(TO) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (VEC == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
  } else {
    p[0] = from_f<TO>(v[0]);
  }
}

template <typename TO, int TAPS, int VEC>
__global__ void __launch_bounds__(128)
conv_silu_kernel(const float* __restrict__ u, int64_t ld, const float* __restrict__ wt, const float* __restrict__ bias, float* __restrict__ state,
                 const int* __restrict__ tiles, int num_decodes, const int* __restrict__ cu_seqlens, const int* __restrict__ context_lens,
                 const int* __restrict__ state_slots, TO* __restrict__ out, int C, int any_taps) {
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  const bool single = (int)blockIdx.x < num_decodes;
  const int b = single ? blockIdx.x : tiles[2 * (blockIdx.x - num_decodes)], i0 = single ? 0 : tiles[2 * (blockIdx.x - num_decodes) + 1];
  const int tok0 = cu_seqlens[b], n = cu_seqlens[b + 1] - tok0, start = context_lens[b] - n, slot = state_slots[b];
  const int taps = TAPS ? TAPS : any_taps, i1 = min(i0 + CS_TILE, n);
  float w[TAPS ? TAPS : 1][VEC], bc[VEC] = {};
  if (c < C) {
    if (TAPS)
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int k = 0; k < VEC; ++k) w[j][k] = wt[(int64_t)(c + k) * TAPS + j];
#pragma unroll
    for (int k = 0; k < VEC; ++k) bc[k] = bias ? bias[c + k] : 0.f;
  }
  pdl_wait();
  pdl_launch_dependents();
  if (c >= C) return;
  float* st = state + (int64_t)(slot < 0 ? 0 : slot) * (taps - 1) * C + c;
  auto input = [&](int i, float (&v)[VEC]) {                   // the input at local index i (negative: before this step)
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = 0.f;
    if (i >= 0) cs_load<VEC>(u + (int64_t)(tok0 + i) * ld + c, v);
    else if (start + i >= 0 && slot >= 0) cs_load<VEC>(st + (int64_t)(i + taps - 1) * C, v);
  };
  auto put = [&](int i, float (&a)[VEC]) {
#pragma unroll
    for (int k = 0; k < VEC; ++k) a[k] = a[k] / (1.f + expf(-a[k]));
    cs_store<VEC>(out + (int64_t)(tok0 + i) * C + c, a);
  };
  if constexpr (TAPS > 0) {
    float x[TAPS][VEC];                                        // x[TAPS - 1] is the current token's
#pragma unroll
    for (int j = 1; j < TAPS; ++j) input(i0 - TAPS + j, x[j]);
    for (int i = i0; i < i1; ++i) {
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
        for (int k = 0; k < VEC; ++k) x[j][k] = x[j + 1][k];
      input(i, x[TAPS - 1]);
      float a[VEC];
#pragma unroll
      for (int k = 0; k < VEC; ++k) a[k] = bc[k];
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int k = 0; k < VEC; ++k) a[k] = fmaf(w[j][k], x[j][k], a[k]);
      put(i, a);
    }
    if (single && slot >= 0)
#pragma unroll
      for (int j = 1; j < TAPS; ++j) cs_store<VEC>(st + (int64_t)(j - 1) * C, x[j]);
  } else {
    for (int i = i0; i < i1; ++i) {
      float a[VEC], x[VEC];
#pragma unroll
      for (int k = 0; k < VEC; ++k) a[k] = bc[k];
      for (int j = 0; j < taps; ++j) {
        input(i - taps + 1 + j, x);
#pragma unroll
        for (int k = 0; k < VEC; ++k) a[k] = fmaf(wt[(int64_t)(c + k) * taps + j], x[k], a[k]);
      }
      put(i, a);
    }
    if (single && slot >= 0)
      for (int j = 1; j < taps; ++j) {                         // (row j - 1 takes what stood in row j: read before it is written over)
        float x[VEC];
        input(j - taps + 1, x);
        cs_store<VEC>(st + (int64_t)(j - 1) * C, x);
      }
  }
}

// The state of the requests from first_req on: the last taps - 1 inputs, in ascending order (see short_conv_state_kernel).
__global__ void __launch_bounds__(256)
conv_silu_state_kernel(const float* __restrict__ u, int64_t ld, float* __restrict__ state, const int* __restrict__ cu_seqlens,
                       const int* __restrict__ context_lens, const int* __restrict__ state_slots, int first_req, int C, int taps) {
  pdl_wait();
  pdl_launch_dependents();
  const int b = first_req + blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  const int slot = state_slots[b], tok0 = cu_seqlens[b], n = cu_seqlens[b + 1] - tok0, start = context_lens[b] - n;
  if (c >= C || slot < 0 || n <= 0) return;
  float* st = state + (int64_t)slot * (taps - 1) * C + c;
  for (int k = 0; k < taps - 1; ++k) {
    const int i = n - (taps - 1) + k;
    float v = 0.f;
    if (i >= 0) v = u[(int64_t)(tok0 + i) * ld + c];
    else if (start + i >= 0) v = st[(int64_t)(i + taps - 1) * C];
    st[(int64_t)k * C] = v;
  }
}

ME_API int me_conv_silu_tile() { return CS_TILE; }

// u: float32, C columns of rows ld elements apart.  wt: [C, taps], bias: [C] float32 or null.  state: [slots, taps - 1, C] float32 (unused with one
// tap).  tiles: [n_tiles, 2] (request, first token) per CS_TILE tokens of the requests from num_decodes on.  out: [T, C] of out_dtype.
ME_API int me_conv_silu(const float* u, int64_t ld, const float* wt, const float* bias, float* state, const int* tiles, int n_tiles, int num_decodes,
                        const int* cu_seqlens, const int* context_lens, const int* state_slots, void* out, int out_dtype, int B, int C, int taps,
                        cudaStream_t stream) {
  if (B == 0 || num_decodes + n_tiles == 0) return 0;
  ME_REQUIRE(C > 0 && taps >= 1 && num_decodes >= 0 && num_decodes <= B, "me_conv_silu: bad sizes B=%d C=%d taps=%d", B, C, taps);
  ME_REQUIRE(taps == 1 || state != nullptr, "me_conv_silu: %d taps need a state", taps);
  auto off = [](const void* p, size_t to) { return p && ((uintptr_t)p % to) != 0; };
  const bool vec = C % 4 == 0 && ld % 4 == 0 && !off(u, 16) && !off(state, 16) && !off(out, out_dtype == ME_F32 ? 16 : 8);
  const int per = vec ? 4 : 1, threads = C / per >= 128 ? 128 : (C / per >= 64 ? 64 : 32);
  const dim3 grid(num_decodes + n_tiles, (C + threads * per - 1) / (threads * per));
  ME_REQUIRE(grid.y <= 65535, "me_conv_silu: too many channels (%d)", C);
#define CS_CASE(TAPS_, VEC_)                                                                                                             \
  me_launch(conv_silu_kernel<TO, TAPS_, VEC_>, grid, dim3(threads), 0, stream, u, ld, wt, bias, state, tiles, num_decodes, cu_seqlens,   \
            context_lens, state_slots, (TO*)out, C, taps)
  ME_DISPATCH_DTYPE(out_dtype, TO, {
    if (vec && taps == 4) CS_CASE(4, 4);
    else if (vec && taps == 3) CS_CASE(3, 4);
    else if (vec && taps == 2) CS_CASE(2, 4);
    else if (vec) CS_CASE(0, 4);
    else if (taps == 4) CS_CASE(4, 1);
    else CS_CASE(0, 1);
  });
#undef CS_CASE
  ME_LAUNCH_CHECK("me_conv_silu");
  if (taps > 1 && num_decodes < B) {
    me_launch(conv_silu_state_kernel, dim3(B - num_decodes, (C + 255) / 256), dim3(256), 0, stream, u, ld, state, cu_seqlens, context_lens,
              state_slots, num_decodes, C, taps);
    ME_LAUNCH_CHECK("me_conv_silu (state)");
  }
  return 0;
}
