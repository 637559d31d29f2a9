// Linear attention whose state decays by one number a head and token, with a state slot per request.
//
// Per head, with q, k of D values, v of V values, a decay a_t in (0, 1] and a factor g_t on what is written:
//   S_t = a_t S_(t-1) + g_t k_t v_t^T              (D x V)
//   o_t = S_t^T q_t + skip * v_t                    (V; ``skip``: a number a head, or none)
// q and k may be shared by groups of neighbouring heads (G groups; head h uses group h / (H / G)).  Two sources of a and g:
//   ``dt`` (the state-space form): g_t = softplus(dt_t + bias), a_t = exp(-exp(a_log) g_t), a column of ``dt`` a head;
//   ``decay`` (a constant a head, with its logarithm ``log2_decay`` in double precision): a = decay, and g_t = k_scale for every token.
// S starts at zero and is float32, as are a, g, their logarithms and all sums; q, k and v are float32 or bfloat16.
//
//   hd_step_kernel         walks a request's tokens one by one, its state in registers: single tokens of a decode step
//   hd_chunk_state_kernel  portions of prompts, HD_LC tokens at a time, all runs of a step side by side: what each run adds,
//                          U = sum_s g_s 2^(B_L - B_s) k_s v_s^T, with B_t the sum of log2 a from the run's first token up to t
//   hd_state_walk_kernel   per request, in order: states[c] <- the state in front of run c; S <- 2^(B_L) S + U_c
//   hd_chunk_out_kernel    o_t = 2^(B_t) q_t^T S_in + sum_{s<=t} (q_t . k_s) g_s 2^(B_t - B_s) v_s + skip v_t
// Every exponent is <= 0.  B is summed and its differences are taken in double precision (64 numbers a run and head), so a decay
// close to 1 behind strong ones keeps its digits.  The first and the last of these three are those of head_decay_mma.cu where bfloat16
// operands and their sizes allow.  The results differ from the token-by-token kernel by the order of sums only.
#include "head_decay.cuh"

template <int N> struct HdVec;
template <> struct HdVec<4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  }
  static __device__ __forceinline__ void load(const bf16* p, float (&v)[4]) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&t.x), b = *reinterpret_cast<const __nv_bfloat162*>(&t.y);
    v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct HdVec<1> {
  template <typename T> static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f<T>(*p); }
  static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
};

// ---- token by token -------------------------------------------------------------------------------------------
// One block = one request x one head x 16 VEC columns of S.  Thread (dy, c): rows dy, dy + 16, ... and VEC columns of S in registers.
template <typename T, int R, int VEC>
__global__ void __launch_bounds__(256) hd_step_kernel(HdArgs a) {
  extern __shared__ __align__(16) float smem[];
  const int D = a.D, V = a.V, D4 = (D + 3) / 4 * 4;      // (what follows starts on 16 bytes)
  float* q_s = smem;                            // [D4]
  float* k_s = q_s + D4;                        // [D4]
  float* parts = k_s + D4;                      // [8][16 VEC]
  const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, c = tid & 15, dy = tid >> 4, warp = tid >> 5, lane = tid & 31;
  const int v0 = (blockIdx.z * 16 + c) * VEC;
  const bool v_ok = v0 < V;                     // (V is a multiple of VEC)
  const int slot = a.slots[b];                  // written by the host, like the lengths
  const int tok0 = a.cu[b], n_tok = a.cu[b + 1] - tok0;
  const bool run = slot >= 0 && n_tok > 0, fresh = a.ctx[b] - n_tok == 0;
  float* Sg = a.S + ((int64_t)(run ? slot : 0) * a.H + h) * D * V + v0;
  float s[R][VEC];
  // (the state is no earlier kernel's business of this step: its loads need not wait for the projections)
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int d = dy + 16 * i;
#pragma unroll
    for (int j = 0; j < VEC; ++j) s[i][j] = 0.f;
    if (run && !fresh && v_ok && d < D) HdVec<VEC>::load(Sg + (int64_t)d * V, s[i]);
  }
  pdl_wait();
  pdl_launch_dependents();
  if (!run) return;
  const int g = h / (a.H / a.G);
  const float skip = a.skip ? a.skip[h] : 0.f;
  for (int i = 0; i < n_tok; ++i) {
    const int64_t t = tok0 + i;
    float gain, decay;
    hd_token(a, t, h, gain, decay);
    const T *qr = reinterpret_cast<const T*>(a.q) + t * a.ldq + (int64_t)g * D, *kr = reinterpret_cast<const T*>(a.k) + t * a.ldk + (int64_t)g * D;
    if (i) __syncthreads();                     // the token before is done with q_s, k_s, parts
    for (int d = tid; d < D; d += 256) {
      q_s[d] = to_f<T>(qr[d]);
      k_s[d] = to_f<T>(kr[d]) * gain;
    }
    float v[VEC] = {}, part[VEC] = {};
    if (v_ok) HdVec<VEC>::load(reinterpret_cast<const T*>(a.v) + t * a.ldv + (int64_t)h * V + v0, v);
    __syncthreads();
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = dy + 16 * r;
      if (d < D) {
        const float qd = q_s[d], kd = k_s[d];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          s[r][j] = fmaf(decay, s[r][j], kd * v[j]);
          part[j] = fmaf(s[r][j], qd, part[j]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) part[j] += __shfl_xor_sync(0xffffffffu, part[j], 16);
    if (lane < 16) HdVec<VEC>::store(parts + (warp * 16 + c) * VEC, part);
    __syncthreads();
    if (dy == 0 && v_ok) {
      float tot[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) tot[j] = skip * v[j];
#pragma unroll
      for (int w = 0; w < 8; ++w)
#pragma unroll
        for (int j = 0; j < VEC; ++j) tot[j] += parts[(w * 16 + c) * VEC + j];
      HdVec<VEC>::store(a.o + t * a.H * V + (int64_t)h * V + v0, tot);
    }
  }
  if (v_ok)
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = dy + 16 * r;
      if (d < D) HdVec<VEC>::store(Sg + (int64_t)d * V, s[r]);
    }
}

// ---- runs of HD_LC tokens -------------------------------------------------------------------------------------
// rows x cols values of a matrix in global memory into shared memory as float32, zeros beyond n_rows and n_cols.
template <typename T, int VEC>
__device__ __forceinline__ void hd_fill(float* dst, int ld_dst, int rows, int cols, const T* src, int64_t ld_src, int n_rows, int n_cols) {
  const int per = cols / VEC;
#pragma unroll 4
  for (int i = threadIdx.x; i < rows * per; i += 256) {
    const int r = i / per, c = (i - r * per) * VEC;
    float v[VEC] = {};
    if (r < n_rows && c < n_cols) HdVec<VEC>::load(src + (int64_t)r * ld_src + c, v);
    HdVec<VEC>::store(dst + r * ld_dst + c, v);
  }
}

// One block = one run x one head x HD_VT columns.  nums[c, h]: the run's numbers.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
hd_chunk_state_kernel(HdArgs a, const int* __restrict__ tiles, float* __restrict__ states, HdRun* __restrict__ nums) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float g_s[HD_LC];
  __shared__ double b_s[HD_LC];
  constexpr int LC = HD_LC, VT = HD_VT;
  const int D = a.D, V = a.V, Dp = (D + 63) / 64 * 64, ldk = Dp + 4;
  float* Kt = smem;                             // [LC][Dp + 4]
  float* Vc = Kt + LC * ldk;                    // [LC][VT], times g_s 2^(B_L - B_s)
  const int tid = threadIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT;
  const int b = tiles[2 * blockIdx.x], q0 = tiles[2 * blockIdx.x + 1];
  const int tok0 = a.cu[b] + q0, L = min(LC, a.cu[b + 1] - tok0);
  pdl_wait();
  pdl_launch_dependents();
  if (L <= 0) return;
  const int g = h / (a.H / a.G);
  hd_run_scalars(a, tok0, L, h, g_s, b_s);
  hd_fill<T, VEC>(Kt, ldk, LC, Dp, reinterpret_cast<const T*>(a.k) + (int64_t)tok0 * a.ldk + (int64_t)g * D, a.ldk, L, D);
  __syncthreads();
  const double bl = b_s[LC - 1];
  if (tid < LC && blockIdx.z == 0) {
    HdRun& run = nums[(int64_t)blockIdx.x * a.H + h];
    run.b[tid] = b_s[tid];
    run.g[tid] = g_s[tid];
  }
  {
    const T* src = reinterpret_cast<const T*>(a.v) + (int64_t)tok0 * a.ldv + (int64_t)h * V + v0;
    constexpr int per = VT / VEC;
#pragma unroll 4
    for (int i = tid; i < LC * per; i += 256) {
      const int r = i / per, c = (i - r * per) * VEC;
      float v[VEC] = {};
      if (r < L && v0 + c < V) HdVec<VEC>::load(src + (int64_t)r * a.ldv + c, v);
      const float f = g_s[r] * exp2f((float)(bl - b_s[r]));
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= f;
      HdVec<VEC>::store(Vc + r * VT + c, v);
    }
  }
  __syncthreads();
  // a thread: rows d0 + 4 ty .. + 3 and columns 4 tx .. + 3; one 16-byte load of each operand a token
  const int ty = tid / 16, tx = tid % 16;
  float* out = states + ((int64_t)blockIdx.x * a.H + h) * D * V;
  for (int d0 = 0; d0 < D; d0 += 64) {
    float acc[4][4] = {};
#pragma unroll 8
    for (int s = 0; s < LC; ++s) {              // (rows beyond L are zero)
      float kk[4], vv[4];
      HdVec<4>::load(Kt + s * ldk + d0 + 4 * ty, kk);
      HdVec<4>::load(Vc + s * VT + 4 * tx, vv);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(kk[i], vv[j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = d0 + 4 * ty + i;
      if (d >= D) continue;
      float* row = out + (int64_t)d * V + v0 + 4 * tx;
      if (VEC == 4) {
        if (v0 + 4 * tx < V) HdVec<4>::store(row, acc[i]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (v0 + 4 * tx + j < V) row[j] = acc[i][j];
      }
    }
  }
}

// One block = one request (first_req + blockIdx.x) x one head x HD_WALK VEC elements of S; a thread walks VEC neighbours.
constexpr int HD_WALK = 128;

template <int VEC>
__global__ void __launch_bounds__(HD_WALK, 8)
hd_state_walk_kernel(HdArgs a, const HdRun* __restrict__ nums, float* states, const int* __restrict__ tiles, int n_tiles, int first_req) {
  __shared__ int first_tile;
  const int b = first_req + blockIdx.x, h = blockIdx.y, DV = a.D * a.V;
  const int e = (blockIdx.z * HD_WALK + threadIdx.x) * VEC;
  const int slot = a.slots[b], tok0 = a.cu[b], n_tok = a.cu[b + 1] - tok0;
  if (threadIdx.x == 0) first_tile = -1;
  __syncthreads();
  for (int i = threadIdx.x; i < n_tiles; i += HD_WALK)           // a request's runs follow one another in the list
    if (tiles[2 * i] == b && tiles[2 * i + 1] == 0) first_tile = i;
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const int c0 = first_tile;
  if (slot < 0 || n_tok <= 0 || c0 < 0 || e >= DV) return;
  float* Sg = a.S + ((int64_t)slot * a.H + h) * DV + e;
  float S[VEC] = {};
  if (a.ctx[b] != n_tok) HdVec<VEC>::load(Sg, S);
  const int n_chunks = (n_tok + HD_LC - 1) / HD_LC;
  const int64_t step = (int64_t)a.H * DV;
  float* st = states + ((int64_t)c0 * a.H + h) * DV + e;
  const HdRun* run = nums + (int64_t)c0 * a.H + h;
  // The loads of the next AHEAD runs are on their way while these runs' states are stored (one group of loads at a time, then its stores,
  // took nearly twice as long: 53 against 29 us for 32 runs of 64 heads of 128 x 64).
  constexpr int AHEAD = 4;
  float u[2][AHEAD][VEC], dec[2][AHEAD];
  auto fetch = [&](int into, int c1) {
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int c = min(c1 + j, n_chunks - 1);
      HdVec<VEC>::load(st + c * step, u[into][j]);
      dec[into][j] = (float)run[(int64_t)c * a.H].b[HD_LC - 1];
    }
  };
  fetch(0, 0);
  for (int pair = 0; pair < n_chunks; pair += 2 * AHEAD) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int c1 = pair + half * AHEAD;
      if (c1 >= n_chunks) break;
      if (c1 + AHEAD < n_chunks) fetch(half ^ 1, c1 + AHEAD);
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        if (c1 + j < n_chunks) {
          HdVec<VEC>::store(st + (c1 + j) * step, S);
          const float f = exp2f(dec[half][j]);
#pragma unroll
          for (int k = 0; k < VEC; ++k) S[k] = fmaf(f, S[k], u[half][j][k]);
        }
      }
    }
  }
  HdVec<VEC>::store(Sg, S);
}

// One block = one run x one head x HD_VT columns; states[c] holds the state in front of the run.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
hd_chunk_out_kernel(HdArgs a, const int* __restrict__ tiles, const float* __restrict__ states, const HdRun* __restrict__ nums) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float g_s[HD_LC];
  __shared__ double b_s[HD_LC];
  constexpr int LC = HD_LC, VT = HD_VT, lda = LC + 4;
  const int D = a.D, V = a.V, D4 = (D + 3) / 4 * 4, ldq = D4 + 4;
  float* Q = smem;                              // [LC][ldq]
  float* K = Q + LC * ldq;                      // [LC][ldq], later the state [D4][VT]
  float* A = K + max(LC * ldq, D4 * VT);        // [LC][lda]
  float* Vs = A + LC * lda;                     // [LC][VT]
  const int tid = threadIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT;
  const int b = tiles[2 * blockIdx.x], q0 = tiles[2 * blockIdx.x + 1];
  const int tok0 = a.cu[b] + q0, L = min(LC, a.cu[b + 1] - tok0);
  pdl_wait();
  pdl_launch_dependents();
  if (L <= 0) return;
  const int g = h / (a.H / a.G);
  if (tid < LC) {
    const HdRun& run = nums[(int64_t)blockIdx.x * a.H + h];
    b_s[tid] = run.b[tid];
    g_s[tid] = run.g[tid];
  }
  hd_fill<T, VEC>(Q, ldq, LC, D4, reinterpret_cast<const T*>(a.q) + (int64_t)tok0 * a.ldq + (int64_t)g * D, a.ldq, L, D);
  hd_fill<T, VEC>(K, ldq, LC, D4, reinterpret_cast<const T*>(a.k) + (int64_t)tok0 * a.ldk + (int64_t)g * D, a.ldk, L, D);
  hd_fill<T, VEC>(Vs, VT, LC, VT, reinterpret_cast<const T*>(a.v) + (int64_t)tok0 * a.ldv + (int64_t)h * V + v0, a.ldv, L, V - v0);
  __syncthreads();
  const int ty = tid / 16, tx = tid % 16;
  {
    float sc[4][4] = {};
    for (int d = 0; d < D4; d += 4) {
      float x[4][4], y[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        HdVec<4>::load(Q + (ty + 16 * i) * ldq + d, x[i]);
        HdVec<4>::load(K + (tx + 16 * i) * ldq + d, y[i]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int k = 0; k < 4; ++k) sc[i][j] = fmaf(x[i][k], y[j][k], sc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = ty + 16 * i, s = tx + 16 * j;
        A[t * lda + s] = s <= t ? sc[i][j] * g_s[s] * exp2f((float)(b_s[t] - b_s[s])) : 0.f;
      }
  }
  __syncthreads();                              // K is read, A is written
  hd_fill<float, VEC>(K, VT, D4, VT, states + ((int64_t)blockIdx.x * a.H + h) * D * V + v0, V, D, V - v0);
  __syncthreads();
  // a thread: rows ty + 16 i and columns 4 tx .. + 3; four terms a turn with 16-byte loads of both operands
  float acc[4][4] = {};
  auto product = [&](const float* X, int ldx, const float* Y, int n) {
    for (int c = 0; c < n; c += 4) {
      float xx[4][4], yy[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) HdVec<4>::load(X + (ty + 16 * i) * ldx + c, xx[i]);
#pragma unroll
      for (int k = 0; k < 4; ++k) HdVec<4>::load(Y + (c + k) * VT + 4 * tx, yy[k]);
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xx[i][k], yy[k][j], acc[i][j]);
    }
  };
  product(Q, ldq, K, D4);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float f = exp2f((float)b_s[ty + 16 * i]);
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] *= f;
  }
  product(A, lda, Vs, LC);
  const float skip = a.skip ? a.skip[h] : 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty + 16 * i;
    if (t >= L) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(skip, Vs[t * VT + 4 * tx + j], acc[i][j]);
    float* row = a.o + (int64_t)(tok0 + t) * a.H * V + (int64_t)h * V + v0 + 4 * tx;
    if (VEC == 4) {
      if (v0 + 4 * tx < V) HdVec<4>::store(row, acc[i]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (v0 + 4 * tx + j < V) row[j] = acc[i][j];
    }
  }
}

int me_head_decay_mma_states(const HdArgs& a, const int* tiles, int n_tiles, float* states, HdRun* nums, cudaStream_t stream);
int me_head_decay_mma_out(const HdArgs& a, const int* tiles, int n_tiles, const float* states, const HdRun* nums, cudaStream_t stream);
bool me_head_decay_mma_takes(const HdArgs& a, int dtype);

template <typename K>
static int hd_raise_smem(K kernel, size_t smem, const char* what) {
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ME_REQUIRE(e == cudaSuccess, "%s: cannot raise shared memory to %zu: %s", what, smem, cudaGetErrorString(e));
  }
  return 0;
}

ME_API int me_head_decay_chunk_len() { return HD_LC; }
ME_API int me_head_decay_run_bytes() { return (int)sizeof(HdRun); }      // what a run and head takes of ``nums_ws``

// q, k: rows of ``dtype`` holding the G groups' D values, ldq / ldk elements apart; v: rows of H heads' V values.  dt: float32 rows of H
// pre-activations with dt_bias, a_log [H], or null with decay [H] and log2_decay [H] (float64).  skip: [H] or null.  S: [slots, H, D, V] float32; o: [T, H*V]
// float32.  Requests [0, num_decodes) are walked token by token.  The others too, unless ``tiles`` ([n_tiles, 2] int32: request and first
// token of every run of HD_LC tokens of the requests from num_decodes on, a request's runs in order and side by side),
// ``states_ws`` ([n_tiles, H, D, V] float32) and ``nums_ws`` (n_tiles * H times me_head_decay_run_bytes, on 16 bytes) are given and D is at most 256.  allow_mma: the
// products of prompts may run on the tensor cores.
ME_API int me_head_decay_scan(const void* q, const void* k, const void* v, int dtype, int64_t ldq, int64_t ldk, int64_t ldv, int H, int G, int D,
                              int V, float k_scale, const float* dt, int64_t ld_dt, const float* dt_bias, const float* a_log,
                              const float* decay, const double* log2_decay, const float* skip, float* S, const int* cu_seqlens, const int* context_lens,
                              const int* state_slots, float* o, int B, int num_decodes, const int* tiles, int n_tiles, float* states_ws,
                              void* nums_ws, int allow_mma, cudaStream_t stream) {
  if (B == 0) return 0;
  ME_REQUIRE(B > 0 && H > 0 && G > 0 && H % G == 0 && D > 0 && V > 0 && H <= 65535 && D <= 1024, "me_head_decay_scan: bad sizes B=%d H=%d G=%d D=%d V=%d", B, H, G, D, V);
  ME_REQUIRE(num_decodes >= 0 && num_decodes <= B, "me_head_decay_scan: %d single-token requests of %d", num_decodes, B);
  ME_REQUIRE(dt ? (dt_bias && a_log) : (decay && log2_decay), "me_head_decay_scan: decays from dt (with its bias and a_log) or constants");
  const HdArgs a = {q, k, v, ldq, ldk, ldv, H, G, D, V, k_scale, dt, ld_dt, dt_bias, a_log, decay, log2_decay, skip, S, cu_seqlens, context_lens, state_slots, o};
  auto off = [](const void* p, size_t to) { return ((uintptr_t)p % to) != 0; };
  const size_t al = dtype == ME_F32 ? 16 : 8;
  const bool out4 = V % 4 == 0 && ldv % 4 == 0 && !off(v, al) && !off(S, 16) && !off(o, 16);
  const size_t D4 = (D + 3) / 4 * 4, Dp = (D + 63) / 64 * 64, v_tiles = (V + HD_VT - 1) / HD_VT;
  const size_t smem_state = sizeof(float) * (HD_LC * (Dp + 4) + HD_LC * HD_VT);
  const size_t lk = HD_LC * (D4 + 4), ls = D4 * HD_VT;
  const size_t smem_out = sizeof(float) * (lk + (lk > ls ? lk : ls) + HD_LC * (HD_LC + 4) + HD_LC * HD_VT);
  const bool chunks = tiles && states_ws && nums_ws && n_tiles > 0 && num_decodes < B && D <= 256 && v_tiles <= 65535 &&
                      ((int64_t)D * V + HD_WALK - 1) / HD_WALK <= 65535 && smem_state <= 220 * 1024 && smem_out <= 220 * 1024;
  const int n_step = chunks ? num_decodes : B;
  if (n_step > 0) {
#define HD_STEP(R_, VEC_)                                                                                                       \
  me_launch(hd_step_kernel<T, R_, VEC_>, dim3(n_step, H, (V + 16 * VEC_ - 1) / (16 * VEC_)), dim3(256),                         \
            sizeof(float) * (2 * D4 + 8 * 16 * VEC_), stream, a)
    ME_DISPATCH_DTYPE(dtype, T, {
      if (out4 && D <= 64) HD_STEP(4, 4);
      else if (out4 && D <= 128) HD_STEP(8, 4);
      else if (out4 && D <= 256) HD_STEP(16, 4);
      else if (D <= 256) HD_STEP(16, 1);
      else HD_STEP(64, 1);
    });
#undef HD_STEP
    ME_LAUNCH_CHECK("me_head_decay_scan (tokens)");
  }
  if (chunks) {
    HdRun* nums = reinterpret_cast<HdRun*>(nums_ws);
    ME_REQUIRE(!off(nums_ws, 16), "me_head_decay_scan: the runs' numbers must start on 16 bytes");
    const bool vec = out4 && D % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && !off(q, al) && !off(k, al) && !off(states_ws, 16);
#define HD_CHUNK(KERNEL_, VEC_, SMEM_, ...)                                                                          \
  do {                                                                                                               \
    if (hd_raise_smem(KERNEL_<T, VEC_>, SMEM_, "me_head_decay_scan")) return 1;                                       \
    me_launch(KERNEL_<T, VEC_>, dim3(n_tiles, H, (unsigned)v_tiles), dim3(256), SMEM_, stream, a, tiles, __VA_ARGS__); \
  } while (0)
    const bool mma = allow_mma && me_head_decay_mma_takes(a, dtype) && !off(states_ws, 16);
    if (mma) {
      if (me_head_decay_mma_states(a, tiles, n_tiles, states_ws, nums, stream)) return 1;
    } else ME_DISPATCH_DTYPE(dtype, T, {
      if (vec) HD_CHUNK(hd_chunk_state_kernel, 4, smem_state, states_ws, nums);
      else HD_CHUNK(hd_chunk_state_kernel, 1, smem_state, states_ws, nums);
    });
    ME_LAUNCH_CHECK("me_head_decay_scan (run states)");
    const bool walk4 = V % 4 == 0 && !off(states_ws, 16) && !off(S, 16);
    const int per = walk4 ? 4 * HD_WALK : HD_WALK;
    const dim3 walk_grid(B - num_decodes, H, (unsigned)(((int64_t)D * V + per - 1) / per));
    if (walk4) me_launch(hd_state_walk_kernel<4>, walk_grid, dim3(HD_WALK), 0, stream, a, (const HdRun*)nums, states_ws, tiles, n_tiles, num_decodes);
    else me_launch(hd_state_walk_kernel<1>, walk_grid, dim3(HD_WALK), 0, stream, a, (const HdRun*)nums, states_ws, tiles, n_tiles, num_decodes);
    ME_LAUNCH_CHECK("me_head_decay_scan (state walk)");
    if (mma) {
      if (me_head_decay_mma_out(a, tiles, n_tiles, states_ws, nums, stream)) return 1;
    } else ME_DISPATCH_DTYPE(dtype, T, {
      if (vec) HD_CHUNK(hd_chunk_out_kernel, 4, smem_out, (const float*)states_ws, (const HdRun*)nums);
      else HD_CHUNK(hd_chunk_out_kernel, 1, smem_out, (const float*)states_ws, (const HdRun*)nums);
    });
#undef HD_CHUNK
    ME_LAUNCH_CHECK("me_head_decay_scan (run outputs)");
  }
  return 0;
}
