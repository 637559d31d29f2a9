// Between the packed projection and the attention of a grouped-query mixer whose projections may have biases and whose
// queries and keys may be normalised on either side of the rotation, or over the whole projection:
//
//   u = W h (+ bias)                                  per head of q (H heads of D), k (G heads of D), v (G heads of Dv)
//   q, k: u <- u / rms(u) * w   (NORM_BEFORE, a weight of D values shared by the heads; q and k have one each)
//   q, k: u <- u / rms(row) * w (NORM_ROW: the root mean square over all heads' values of the token's q, or of its k, and a
//         weight for every one of them)
//   q, k: rotary positions on the first ``rot`` elements of a head, element i paired with element i + rot/2:
//         (a, b) -> (a cos t - b sin t, b cos t + a sin t), t = position * freq[i]; the angle is formed in double precision
//         from the int32 position and a table of rot/2 frequencies (so any scaling of the frequencies is the table's
//         business), brought into [-pi, pi] there, then float32 sine and cosine, both times rot_mag
//   q, k: u <- u / rms(u)       (NORM_AFTER, no weight)
//   q: u <- u * q_scale[head]   (a learned number per query head that multiplies the head's scores; optional)
//   q: u <- u * (1 + temp_coef ln(floor((position + 1) / temp_every) + 1))      (a temperature that grows with the position)
//   v: u <- u * v_scale
//   q -> q_out [T, heads, q_row]; k, v -> the paged cache rows that slot_mapping names ([page][keys | values][kv head][offset][HD])
//
// With ``maps`` M = 2 every head of q and k has two maps of D elements side by side (two sets of scores over the same values):
// the columns are q (H heads of M x D), k (G heads of M x D), v (G heads of Dv), and each map is normalised and rotated by itself.
// The cache row of a key holds its maps one after the other; every query map gets a row of q_out of its own, its values where
// that map lies in a key's row and zeros elsewhere, so that its product with a whole key row is its map's score.  Rows of
// q_out and of the cache that are longer than what they hold are filled with zeros.
//
// With ``own_kv`` 0 the rows hold queries only (a mixer that reads another layer's keys and values) and nothing is written
// to the cache.  rms(u) = sqrt(mean(u^2) + eps).  Everything is float32 until the stores.  Where sizes and pointers allow four
// values at a time a block takes a token and holds its whole row in registers (attn_prep_vec_kernel); else one warp = one map of one
// head of one token, and with NORM_ROW a block takes a token, so that the sums over the whole projection are taken once.
#include "common.cuh"

constexpr int AP_MAX = 256;     // largest head
constexpr int AP_VEC_MIN_TOKENS = 128;

enum { AP_NORM_NONE = 0, AP_NORM_BEFORE = 1, AP_NORM_AFTER = 2, AP_NORM_ROW = 3 };

struct PrepArgs {
  const float* proj;
  int64_t ld;
  const float* bias;
  const float *q_w, *k_w;
  int norm_mode;
  float eps;
  const double* freq;
  int rot;
  const int* positions;
  const int* slot_mapping;
  int HD, page_size, H, G, D, Dv, M, q_row, n_tok;
  const float* q_scale;
  int own_kv;
  float temp_coef, temp_every, v_scale, rot_mag;
};

// One unit of a token's row: hs counts the query maps, then the key maps, then the value heads.  inv_q, inv_k: 1 / rms of the
// token's whole q and k (NORM_ROW only).
template <typename T>
__device__ __forceinline__ void prep_unit(const PrepArgs& a, T* __restrict__ q_out, T* __restrict__ pool, float* st, int t, int hs, int lane,
                                          float inv_q, float inv_k) {
  const int D = a.D, M = a.M, HM = a.H * M, GM = a.G * M;
  const bool is_q = hs < HM, is_k = !is_q && hs < HM + GM;
  const int unit = is_q ? hs : (is_k ? hs - HM : hs - HM - GM);        // (head, map), or the value head
  const int head = (is_q || is_k) ? unit / M : unit, map = (is_q || is_k) ? unit - head * M : 0;
  const int n = (is_q || is_k) ? D : a.Dv;
  const int col0 = is_q ? unit * D : (is_k ? HM * D + unit * D : (HM + GM) * D + unit * a.Dv);
  const float* src = a.proj + (int64_t)t * a.ld + col0;
  float u[AP_MAX / 32];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < AP_MAX / 32; ++i) {
    const int d = lane + 32 * i;
    u[i] = d < n ? src[d] + (a.bias ? a.bias[col0 + d] : 0.f) : 0.f;
    ss = fmaf(u[i], u[i], ss);
  }
  if (is_q || is_k) {
    if (a.norm_mode == AP_NORM_BEFORE || a.norm_mode == AP_NORM_ROW) {
      const bool whole = a.norm_mode == AP_NORM_ROW;
      const float r = whole ? (is_q ? inv_q : inv_k) : 1.0f / sqrtf(warp_sum(ss) / (float)D + a.eps);
      const float* w = (is_q ? a.q_w : a.k_w) + (whole ? unit * D : 0);
#pragma unroll
      for (int i = 0; i < AP_MAX / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < D) u[i] = u[i] * r * w[d];
      }
    }
    if (a.rot > 0) {
#pragma unroll
      for (int i = 0; i < AP_MAX / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < D) st[d] = u[i];
      }
      __syncwarp();
      const int half = a.rot / 2;
      const double pos = (double)a.positions[t];
#pragma unroll
      for (int i = 0; i < AP_MAX / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < a.rot) {
          const int f = d < half ? d : d - half;
          float sn, cs;
          double x = pos * a.freq[f];
          x -= 6.283185307179586476925 * rint(x * 0.15915494309189533577);
          sincosf((float)x, &sn, &cs);
          sn *= a.rot_mag;
          cs *= a.rot_mag;
          u[i] = d < half ? st[d] * cs - st[d + half] * sn : st[d] * cs + st[d - half] * sn;
        }
      }
      __syncwarp();                                    // (the warp may take another unit)
    }
    if (a.norm_mode == AP_NORM_AFTER) {
      ss = 0.f;
#pragma unroll
      for (int i = 0; i < AP_MAX / 32; ++i) ss = fmaf(u[i], u[i], ss);
      const float r = 1.0f / sqrtf(warp_sum(ss) / (float)D + a.eps);
#pragma unroll
      for (int i = 0; i < AP_MAX / 32; ++i) u[i] *= r;
    }
    if (is_q && a.q_scale) {
      const float f = a.q_scale[head];
#pragma unroll
      for (int i = 0; i < AP_MAX / 32; ++i) u[i] *= f;
    }
    if (is_q && a.temp_every > 0.f) {
      const float f = fmaf(a.temp_coef, logf(floorf((float)(a.positions[t] + 1) / a.temp_every) + 1.0f), 1.0f);
#pragma unroll
      for (int i = 0; i < AP_MAX / 32; ++i) u[i] *= f;
    }
  } else {
#pragma unroll
    for (int i = 0; i < AP_MAX / 32; ++i) u[i] *= a.v_scale;
  }
  // the row that takes the unit, where in it the unit's values start, and which of its elements this warp fills with zeros
  T* dst;
  int base = map * D, zero_lo, zero_hi;
  if (is_q) {
    dst = q_out + ((int64_t)t * HM + unit) * a.q_row;
    zero_lo = 0;
    zero_hi = a.q_row;
  } else {
    const int slot = a.slot_mapping ? a.slot_mapping[t] : -1;
    if (slot < 0) return;
    const int page = slot / a.page_size, off = slot - page * a.page_size;
    dst = pool + ((((int64_t)page * 2 + (is_k ? 0 : 1)) * a.G + head) * a.page_size + off) * a.HD;
    zero_lo = base;                                    // what lies behind the last map (or the value)
    zero_hi = map == (is_k ? M - 1 : 0) ? a.HD : 0;
  }
#pragma unroll
  for (int i = 0; i < AP_MAX / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < n) dst[base + d] = from_f<T>(u[i]);
  }
  for (int d = zero_lo + lane; d < zero_hi; d += 32)
    if (d < base || d >= base + n) dst[d] = from_f<T>(0.f);
}

template <typename T>
__global__ void __launch_bounds__(128) attn_prep_kernel(PrepArgs a, T* __restrict__ q_out, T* __restrict__ pool) {
  __shared__ float stage[4][AP_MAX];
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int per_tok = a.H * a.M + (a.own_kv ? a.G * (a.M + 1) : 0);
  const int64_t unit = (int64_t)blockIdx.x * 4 + warp;
  if (unit >= (int64_t)a.n_tok * per_tok) return;
  const int t = (int)(unit / per_tok);
  prep_unit<T>(a, q_out, pool, stage[warp], t, (int)(unit - (int64_t)t * per_tok), lane, 1.f, 1.f);
}

// A token a block: the sums over the whole q and the whole k first, then the units.
template <typename T>
__global__ void __launch_bounds__(256) attn_prep_row_kernel(PrepArgs a, T* __restrict__ q_out, T* __restrict__ pool) {
  __shared__ float stage[8][AP_MAX];
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nq = a.H * a.M * a.D, nk = a.own_kv ? a.G * a.M * a.D : 0;
  const float* row = a.proj + (int64_t)t * a.ld;
  float sq = 0.f, sk = 0.f;
#pragma unroll 4
  for (int c = threadIdx.x; c < nq; c += 256) {
    const float u = row[c] + (a.bias ? a.bias[c] : 0.f);
    sq = fmaf(u, u, sq);
  }
#pragma unroll 4
  for (int c = nq + threadIdx.x; c < nq + nk; c += 256) {
    const float u = row[c] + (a.bias ? a.bias[c] : 0.f);
    sk = fmaf(u, u, sk);
  }
  const float inv_q = 1.0f / sqrtf(block_sum(sq, red) / (float)nq + a.eps);
  const float inv_k = nk ? 1.0f / sqrtf(block_sum(sk, red) / (float)nk + a.eps) : 0.f;
  const int per_tok = a.H * a.M + (a.own_kv ? a.G * (a.M + 1) : 0);
  for (int hs = warp; hs < per_tok; hs += 8) prep_unit<T>(a, q_out, pool, stage[warp], t, hs, lane, inv_q, inv_k);
}

template <typename T> struct Four;
template <> struct Four<float> {
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Four<bf16> {
  static __device__ __forceinline__ void store(bf16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
  }
};
template <int LANES> __device__ __forceinline__ float lanes_sum(float x) {
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
  return x;
}

// A token a block, four neighbouring values a thread, LANES threads a unit (a map of a query or key head; 4 LANES elements of a
// value head) and up to PASSES units a thread: the token's whole row is in registers after one round of loads.  The rotation's
// cosines and sines are formed once a token.  Takes D up to 4 LANES, and D, Dv, rot / 2, the rows' lengths and the pointers as
// multiples of four values.
template <typename T, int LANES, int PASSES>
__global__ void __launch_bounds__(256) attn_prep_vec_kernel(PrepArgs a, T* __restrict__ q_out, T* __restrict__ pool) {
  constexpr int SLOTS = 256 / LANES, WIDTH = 4 * LANES;
  __shared__ float cs_s[WIDTH / 2], sn_s[WIDTH / 2], red[32];
  const int t = blockIdx.x, tid = threadIdx.x, l = tid % LANES, e = 4 * l, lane = tid & 31;
  const int D = a.D, Dv = a.Dv, M = a.M, HM = a.H * M, GM = a.own_kv ? a.G * M : 0;
  const int chunks = (Dv + WIDTH - 1) / WIDTH, units = HM + GM + (a.own_kv ? a.G * chunks : 0);
  const int half = a.rot / 2, pos = a.positions[t], slot = a.slot_mapping ? a.slot_mapping[t] : -1;       // (written by the host)
  if (tid < half) {
    double x = (double)pos * a.freq[tid];
    x -= 6.283185307179586476925 * rint(x * 0.15915494309189533577);
    float sn, cs;
    sincosf((float)x, &sn, &cs);
    sn_s[tid] = sn * a.rot_mag;
    cs_s[tid] = cs * a.rot_mag;
  }
  pdl_wait();
  pdl_launch_dependents();
  const float* row = a.proj + (int64_t)t * a.ld;
  float u[PASSES][4];
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const int hs = p * SLOTS + tid / LANES;
    const int v = hs - HM - GM, head = v / chunks, at = (v - head * chunks) * WIDTH + e;
    const bool on = hs < units && (v < 0 ? e < D : at < Dv);
    const int col = v < 0 ? hs * D + e : (HM + GM) * D + head * Dv + at;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on) {
      x = *reinterpret_cast<const float4*>(row + col);
      if (a.bias) {
        const float4 b = *reinterpret_cast<const float4*>(a.bias + col);
        x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
      }
    }
    u[p][0] = x.x; u[p][1] = x.y; u[p][2] = x.z; u[p][3] = x.w;
  }
  float inv_q = 1.f, inv_k = 1.f;
  if (a.norm_mode == AP_NORM_ROW) {
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int p = 0; p < PASSES; ++p) {
      const int hs = p * SLOTS + tid / LANES;
      const float s = fmaf(u[p][0], u[p][0], u[p][1] * u[p][1]) + fmaf(u[p][2], u[p][2], u[p][3] * u[p][3]);
      if (hs < HM) sq += s;
      else if (hs < HM + GM) sk += s;
    }
    inv_q = 1.0f / sqrtf(block_sum(sq, red) / (float)(HM * D) + a.eps);
    if (GM) inv_k = 1.0f / sqrtf(block_sum(sk, red) / (float)(GM * D) + a.eps);
  } else if (half > 0) {
    __syncthreads();                                   // the cosines and sines are in place
  }
  const float temp = a.temp_every > 0.f ? fmaf(a.temp_coef, logf(floorf((float)(pos + 1) / a.temp_every) + 1.0f), 1.0f) : 1.0f;
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    if (p * SLOTS >= units) break;                     // (the same in all threads)
    const int hs = p * SLOTS + tid / LANES;
    const bool is_q = hs < HM, qk = hs < HM + GM;
    if (a.norm_mode == AP_NORM_BEFORE || a.norm_mode == AP_NORM_ROW) {
      const bool whole = a.norm_mode == AP_NORM_ROW;
      float r = is_q ? inv_q : inv_k;
      if (!whole) r = 1.0f / sqrtf(lanes_sum<LANES>(fmaf(u[p][0], u[p][0], u[p][1] * u[p][1]) + fmaf(u[p][2], u[p][2], u[p][3] * u[p][3])) / (float)D + a.eps);
      if (qk && e < D) {
        const float4 w = *reinterpret_cast<const float4*>((is_q ? a.q_w : a.k_w) + (whole ? (is_q ? hs : hs - HM) * D : 0) + e);
        u[p][0] = u[p][0] * r * w.x; u[p][1] = u[p][1] * r * w.y; u[p][2] = u[p][2] * r * w.z; u[p][3] = u[p][3] * r * w.w;
      }
    }
    if (half > 0) {
      const int mate = lane + (e < half ? half / 4 : -(half / 4));          // the lane that holds the other element of each pair
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float o = __shfl_sync(0xffffffffu, u[p][j], mate & 31);
        if (qk && e < a.rot) {
          const int f = (e < half ? e : e - half) + j;
          u[p][j] = e < half ? u[p][j] * cs_s[f] - o * sn_s[f] : u[p][j] * cs_s[f] + o * sn_s[f];
        }
      }
    }
    if (a.norm_mode == AP_NORM_AFTER) {
      const float r = 1.0f / sqrtf(lanes_sum<LANES>(fmaf(u[p][0], u[p][0], u[p][1] * u[p][1]) + fmaf(u[p][2], u[p][2], u[p][3] * u[p][3])) / (float)D + a.eps);
      if (qk)
#pragma unroll
        for (int j = 0; j < 4; ++j) u[p][j] *= r;
    }
    if (hs >= units) continue;                         // (no shuffle from here on)
    if (qk) {
      const int unit = is_q ? hs : hs - HM, head = unit / M, map = unit - head * M, base = map * D;
      T* dst;
      int zero_lo, zero_hi;
      if (is_q) {
        const float f = temp * (a.q_scale ? a.q_scale[head] : 1.0f);
#pragma unroll
        for (int j = 0; j < 4; ++j) u[p][j] *= f;
        dst = q_out + ((int64_t)t * HM + unit) * a.q_row;
        zero_lo = 0;
        zero_hi = a.q_row;
      } else {
        if (slot < 0) continue;
        const int page = slot / a.page_size, off = slot - page * a.page_size;
        dst = pool + ((((int64_t)page * 2) * a.G + head) * a.page_size + off) * a.HD;
        zero_lo = base;
        zero_hi = map == M - 1 ? a.HD : 0;
      }
      if (e < D) Four<T>::store(dst + base + e, u[p]);
      const float none[4] = {0.f, 0.f, 0.f, 0.f};
      for (int d = zero_lo + e; d < zero_hi; d += WIDTH)
        if (d < base || d >= base + D) Four<T>::store(dst + d, none);
    } else {
      if (slot < 0) continue;
      const int v = hs - HM - GM, head = v / chunks, chunk = v - head * chunks, at = chunk * WIDTH + e;
      const int page = slot / a.page_size, off = slot - page * a.page_size;
      T* dst = pool + ((((int64_t)page * 2 + 1) * a.G + head) * a.page_size + off) * a.HD;
#pragma unroll
      for (int j = 0; j < 4; ++j) u[p][j] = at < Dv ? u[p][j] * a.v_scale : 0.f;
      for (int d = at; d < a.HD && (d == at || chunk == chunks - 1); d += WIDTH) {      // the last chunk fills the row up
        Four<T>::store(dst + d, u[p]);
#pragma unroll
        for (int j = 0; j < 4; ++j) u[p][j] = 0.f;
      }
    }
  }
}

// Whether the kernel above takes the launch, and with how many lanes a unit and passes (0: no).  Steps of few tokens without NORM_ROW
// stay with a warp a unit, which spreads a token's heads over the SMs (32 heads of 128, 1 to 64 tokens: 8 to 10 us against 11 to 12 with
// its launch; 256 tokens: 14 against 12, 2,048: 61 against 35).
static int prep_vec_passes(const PrepArgs& a, const void* q_out, const void* pool, int dtype, int& lanes) {
  auto off = [](const void* p, size_t to) { return p && ((uintptr_t)p % to) != 0; };
  const size_t al = dtype == ME_F32 ? 16 : 8;
  lanes = a.D <= 64 ? 16 : 32;
  if (a.n_tok < AP_VEC_MIN_TOKENS && a.norm_mode != AP_NORM_ROW) return 0;
  if (a.D % 4 || a.Dv % 4 || a.rot % 8 || a.D > 128 || a.ld % 4 || a.q_row % 4 || a.HD % 4 || off(a.proj, 16) || off(a.bias, 16) || off(a.q_w, 16) ||
      off(a.k_w, 16) || off(q_out, al) || off(pool, al))
    return 0;
  const int chunks = (a.Dv + 4 * lanes - 1) / (4 * lanes), units = a.H * a.M + (a.own_kv ? a.G * (a.M + chunks) : 0);
  const int passes = (units + 256 / lanes - 1) / (256 / lanes);
  return passes <= 3 ? 3 : (passes <= 6 ? 6 : (passes <= 12 ? 12 : 0));
}

// proj: [T, ld] float32 rows holding q (H*M*D), k (G*M*D), v (G*Dv) in their first columns, M = maps.  bias: a float32 value for
// each of these columns or null.  q_w, k_w: [D] float32 (NORM_BEFORE), [H*M*D] and [G*M*D] (NORM_ROW).  freq: [rot/2] float64 or
// null with rot 0.  slot_mapping: [T] int32 cache rows (page * page_size + offset;
// negative: not written) or null (no keys and values are written).  q_scale: [H] float32 or null.  own_kv 0: the rows hold the
// query columns only.  q_out: [T, H*M, q_row].  temp_every 0: no temperature.
ME_API int me_attn_prep(const float* proj, int64_t ld, const float* bias, const float* q_w, const float* k_w, int norm_mode,
                        float eps, const double* freq, int rot, const int* positions, const int* slot_mapping,
                        void* q_out, int q_row, void* pool, int dtype, int HD, int page_size, int H, int G, int D, int Dv, int maps, int T,
                        const float* q_scale, int own_kv, float temp_coef, float temp_every, float v_scale, float rot_mag,
                        cudaStream_t stream) {
  if (T == 0) return 0;
  ME_REQUIRE(T > 0 && H > 0 && G > 0 && D >= 1 && D <= AP_MAX && Dv >= 1 && Dv <= AP_MAX && (maps == 1 || maps == 2),
             "me_attn_prep: bad sizes H=%d G=%d D=%d Dv=%d maps=%d", H, G, D, Dv, maps);
  ME_REQUIRE(rot >= 0 && rot <= D && rot % 2 == 0 && (rot == 0 || freq), "me_attn_prep: %d of %d elements cannot be rotated", rot, D);
  ME_REQUIRE((norm_mode != AP_NORM_BEFORE && norm_mode != AP_NORM_ROW) || (q_w && (k_w || !own_kv)), "me_attn_prep: a weighted norm needs its weights");
  ME_REQUIRE(q_row >= maps * D, "me_attn_prep: query rows of %d elements are too short", q_row);
  ME_REQUIRE(!slot_mapping || (pool && HD >= maps * D && HD >= Dv), "me_attn_prep: cache rows of %d elements are too short", HD);
  ME_REQUIRE(temp_every >= 0.f, "me_attn_prep: the temperature's step must not be negative");
  const PrepArgs a = {proj, ld, bias, q_w, k_w, norm_mode, eps, freq, rot, positions, slot_mapping, HD, page_size, H, G, D, Dv, maps,
                      q_row, T, q_scale, own_kv, temp_coef, temp_every, v_scale, rot_mag};
  const int64_t units = (int64_t)T * (H * maps + (own_kv ? G * (maps + 1) : 0));
  int lanes = 0;
  const int passes = prep_vec_passes(a, q_out, pool, dtype, lanes);
  if (passes) {
#define AP_VEC(LANES_, PASSES_)                                                                                                       \
  if (lanes == LANES_ && passes == PASSES_)                                                                                           \
    me_launch(attn_prep_vec_kernel<TT, LANES_, PASSES_>, dim3(T), dim3(256), 0, stream, a, (TT*)q_out, (TT*)pool)
    ME_DISPATCH_DTYPE(dtype, TT, {
      AP_VEC(16, 3); AP_VEC(16, 6); AP_VEC(16, 12);
      AP_VEC(32, 3); AP_VEC(32, 6); AP_VEC(32, 12);
    });
#undef AP_VEC
    ME_LAUNCH_CHECK("me_attn_prep");
    return 0;
  }
  ME_DISPATCH_DTYPE(dtype, TT, {
    if (norm_mode == AP_NORM_ROW) me_launch(attn_prep_row_kernel<TT>, dim3(T), dim3(256), 0, stream, a, (TT*)q_out, (TT*)pool);
    else me_launch(attn_prep_kernel<TT>, dim3((unsigned)((units + 3) / 4)), dim3(128), 0, stream, a, (TT*)q_out, (TT*)pool);
  });
  ME_LAUNCH_CHECK("me_attn_prep");
  return 0;
}
