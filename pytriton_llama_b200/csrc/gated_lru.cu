// The gated linear recurrence of a block of channels: with u the convolution's result and zr, zi the blocks' products of it,
//
//   r = sigmoid(zr + b_r),  i = sigmoid(zi + b_i),  log a = -rate r   (rate = decay limit * softplus(lam) per channel)
//   S <- a S + sqrt(1 - a^2) i u,      out = S * gelu_tanh(y + b_y) * scale
//
// All float32.  The decay is kept as e = a - 1 = expm1(log a) and applied as S + (e S + ...): a channel that hardly decays would
// lose the low bits of 1 - a, and with them a systematic share of its memory, if a were rounded.  1 - a^2 = -e (2 + e).
//
// gated_lru_scan, zr and zi given (products of many tokens, or float32): a block owns kLruChannels neighbouring channels
// of one request; its NG groups of as many threads take kLruTokens tokens each of a tile of NG * kLruTokens.  Every group folds its
// tokens into (product of a, less one; result from zero), these meet in shared memory, every group folds those before its own onto
// the state and walks its tokens once more.  So a tile's loads are in flight together, and only the tiles follow one another.  The fold's
// grouping depends on the place of a token within its portion, the arithmetic is a chain of fused multiply-adds either way.
//
// gated_lru_single, one token per request, 16-bit: a warp per channel reads its two weight rows once and every token's block of
// u, and lane t finishes token t: products, gates, state and output in one kernel.
//
// The state of a request is read from its slot unless the portion starts at position 0.
#include "common.cuh"

namespace ptl {

constexpr int kLruTokens = 8;       // tokens of a group per tile
constexpr int kLruChannels = 16;    // channels of a block (half a warp: a real model's few thousand channels then fill the SMs)

struct LruArgs {
  void* out;                        // rows of out_ld elements, results at `column`
  const void *u, *y;                // [T, n]; y rows of y_ld
  const float *gate_bias, *rate, *y_bias;     // [2, n] (r, then i), [n], [n]
  float* state;                     // [slots, n]
  const int *q_start, *positions, *state_slot;
  int n, out_ld, column, y_ld;
  float scale;
};

// FAST (16-bit inputs): the fast exponential and quotient, off by about |z| * 2^-23, beside inputs rounded to 2^-9.  The decay
// itself is always worked out in full.
template <bool FAST>
__device__ __forceinline__ float lru_sigmoid(float z) {
  return FAST ? __fdividef(1.0f, 1.0f + __expf(-z)) : 1.0f / (1.0f + expf(-z));
}
// 0.5 z (1 + tanh(v)) = z sigmoid(2 v), v = sqrt(2/pi) (z + 0.044715 z^3)
template <bool FAST>
__device__ __forceinline__ float lru_gelu(float z) {
  const float v = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return FAST ? z * lru_sigmoid<true>(2.0f * v) : 0.5f * z * (1.0f + tanhf(v));
}
// a - 1 and what enters the state
template <bool FAST>
__device__ __forceinline__ void lru_gates(float zr, float zi, float rate, float u, float& e, float& add) {
  e = expm1f(-rate * lru_sigmoid<FAST>(zr));
  add = sqrtf(-e * (2.0f + e)) * lru_sigmoid<FAST>(zi) * u;
}
// a S + add
__device__ __forceinline__ float lru_step(float e, float S, float add) { return S + fmaf(e, S, add); }

// Channel c of block b = c / s: its zr at z + b * z_block + t * z_tok + c % s, its zi s further on.
template <typename T, int NG>
__global__ void __launch_bounds__(NG * kLruChannels)
gated_lru_scan_kernel(const float* __restrict__ z, long long z_block, long long z_tok, int s, const LruArgs p) {
  __shared__ float s_e[2][NG][kLruChannels], s_b[2][NG][kLruChannels];
  pdl_wait();
  pdl_launch_dependents();
  const int r = blockIdx.y;
  const int lo = p.q_start[r], hi = p.q_start[r + 1];
  if (hi <= lo || p.state_slot[r] < 0) return;
  const int lane = threadIdx.x % kLruChannels, grp = threadIdx.x / kLruChannels;
  const bool live = blockIdx.x * kLruChannels + lane < p.n;
  const int c = live ? blockIdx.x * kLruChannels + lane : p.n - 1;       // lanes past the end shadow the last channel and store nothing
  const float* zc = z + (long long)(c / s) * z_block + c % s;
  const T* u = (const T*)p.u + c;
  const T* y = (const T*)p.y + c;
  T* out = (T*)p.out + p.column + c;
  const float br = p.gate_bias[c], bi = p.gate_bias[p.n + c], rate = p.rate[c], by = p.y_bias[c];
  float* st = p.state + (size_t)p.state_slot[r] * p.n + c;
  float S = p.positions[lo] == 0 ? 0.f : *st;
  float zr[kLruTokens], zi[kLruTokens];
  T ru[kLruTokens], ry[kLruTokens];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < kLruTokens; ++k) {
      const int t = min(t0 + grp * kLruTokens + k, hi - 1);
      zr[k] = zc[t * z_tok];
      zi[k] = zc[t * z_tok + s];
      ru[k] = u[(size_t)t * p.n];
      ry[k] = y[(size_t)t * p.y_ld];
    }
  };
  fetch(lo);
  int buf = 0;
  for (int t0 = lo; t0 < hi; t0 += NG * kLruTokens, buf ^= 1) {
    const int first = t0 + grp * kLruTokens;
    float e[kLruTokens], add[kLruTokens], g[kLruTokens];
    float E = 0.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < kLruTokens; ++k) {
      lru_gates<sizeof(T) == 2>(zr[k] + br, zi[k] + bi, rate, to_f32(ru[k]), e[k], add[k]);
      if (first + k >= hi) { e[k] = 0.f; add[k] = 0.f; }       // past the end: nothing changes
      g[k] = lru_gelu<sizeof(T) == 2>(to_f32(ry[k]) + by) * p.scale;
      E = lru_step(e[k], E, e[k]);
      B = lru_step(e[k], B, add[k]);
    }
    if (t0 + NG * kLruTokens < hi) fetch(t0 + NG * kLruTokens);        // in flight while the tile is folded and walked
    s_e[buf][grp][lane] = E;
    s_b[buf][grp][lane] = B;
    __syncthreads();                                         // (the other buffer may still be read by groups behind)
    float mine = S;
#pragma unroll
    for (int w = 0; w < NG; ++w) {
      if (w == grp) mine = S;
      S = lru_step(s_e[buf][w][lane], S, s_b[buf][w][lane]);
    }
#pragma unroll
    for (int k = 0; k < kLruTokens; ++k) {
      mine = lru_step(e[k], mine, add[k]);
      if (live && first + k < hi) out[(size_t)(first + k) * p.out_ld] = from_f32<T>(mine * g[k]);
    }
  }
  if (live && grp == 0) *st = S;
}

constexpr int kLruSingleTokens = 32;   // tokens of a step that gated_lru_single takes at most (a lane each)

// w rows [blocks][2 s][s]: the r rows of a block, then its i rows.  Token t is the only one of request tok_req[t].
__global__ void __launch_bounds__(256)
gated_lru_single_kernel(const __nv_bfloat16* __restrict__ w, int s, const int* __restrict__ tok_req, int tokens, const LruArgs p) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c = blockIdx.x * 8 + warp;
  if (c >= p.n) return;
  const int b = c / s, e = c % s;
  const __nv_bfloat16* wr = w + ((size_t)b * 2 * s + e) * s;
  const __nv_bfloat16* wi = wr + (size_t)s * s;
  const __nv_bfloat16* ub = (const __nv_bfloat16*)p.u + (size_t)b * s;
  float zr = 0.f, zi = 0.f;                 // lane t: token t
  // the row is walked in slabs of 256 entries, 8 neighbours a lane; the weights depend on no earlier kernel
  bool waited = false;
  for (int k0 = 0; k0 < s; k0 += 256) {
    const int k = k0 + lane * 8;
    float fr[8], fi[8];
    if (k < s) {
      const Vec16<__nv_bfloat16> a = load16(wr + k), d = load16(wi + k);
#pragma unroll
      for (int x = 0; x < 8; ++x) { fr[x] = a.get(x); fi[x] = d.get(x); }
    } else {
#pragma unroll
      for (int x = 0; x < 8; ++x) fr[x] = fi[x] = 0.f;
    }
    if (!waited) {
      pdl_wait();
      pdl_launch_dependents();
      waited = true;
    }
    for (int t = 0; t < tokens; ++t) {
      float pr = 0.f, pi = 0.f;
      if (k < s) {
        const Vec16<__nv_bfloat16> v = load16(ub + (size_t)t * p.n + k);
#pragma unroll
        for (int x = 0; x < 8; ++x) {
          pr = fmaf(fr[x], v.get(x), pr);
          pi = fmaf(fi[x], v.get(x), pi);
        }
      }
      pr = warp_sum(pr);
      pi = warp_sum(pi);
      if (lane == t) { zr += pr; zi += pi; }
    }
  }
  if (lane >= tokens) return;
  const int r = tok_req[lane];
  if (r < 0 || p.state_slot[r] < 0) return;
  float less, add;
  lru_gates<true>(zr + p.gate_bias[c], zi + p.gate_bias[p.n + c], p.rate[c], __bfloat162float(ub[(size_t)lane * p.n + e]), less, add);
  float* st = p.state + (size_t)p.state_slot[r] * p.n + c;
  const float S = lru_step(less, p.positions[lane] == 0 ? 0.f : *st, add);
  *st = S;
  const float g = lru_gelu<true>(__bfloat162float(((const __nv_bfloat16*)p.y)[(size_t)lane * p.y_ld + c]) + p.y_bias[c]) * p.scale;
  ((__nv_bfloat16*)p.out)[(size_t)lane * p.out_ld + p.column + c] = __float2bfloat16_rn(S * g);
}

inline int lru_check(const LruArgs& p, int s) {
  PTL_REQUIRE(p.n > 0 && s > 0 && p.n % s == 0 && p.column >= 0 && p.column + p.n <= p.out_ld && p.n <= p.y_ld,
              "gated_lru: bad sizes channels=%d block=%d", p.n, s);
  return 0;
}

template <typename T>
int gated_lru_scan(const float* z, long long z_block, long long z_tok, int s, const LruArgs& p, int requests, int longest, void* stream) {
  if (int rc = lru_check(p, s)) return rc;
  PTL_REQUIRE(requests >= 0 && requests <= 65535 && z_tok >= 2 * s && z_block >= 0, "gated_lru: bad sizes of the blocks' products");
  if (requests == 0) return 0;
  const dim3 grid((p.n + kLruChannels - 1) / kLruChannels, requests);
#define PTL_LRU(NG) return launch_kernel("gated_lru_scan", gated_lru_scan_kernel<T, NG>, grid, dim3(NG * kLruChannels), 0, as_stream(stream), z, z_block, \
                                         z_tok, s, p)
  if (longest <= 2 * kLruTokens) PTL_LRU(2);
  if (longest <= 8 * kLruTokens) PTL_LRU(8);
  PTL_LRU(32);
#undef PTL_LRU
}

}  // namespace ptl

#define PTL_GATED_LRU(SUFFIX, TYPE)                                                                                              \
  PTL_EXPORT int ptl_gated_lru_scan##SUFFIX(void* out, int out_ld, int column, const void* u, const float* z, long long z_block,  \
                                            long long z_tok, int s, const float* gate_bias, const float* rate, const void* y,    \
                                            int y_ld, const float* y_bias, float* state, const int* q_start,                     \
                                            const int* positions, const int* state_slot, int requests, int longest, int n,       \
                                            float scale, void* stream) {                                                         \
    const ptl::LruArgs p = {out, u, y, gate_bias, rate, y_bias, state, q_start, positions, state_slot, n, out_ld, column, y_ld, scale}; \
    return ptl::gated_lru_scan<TYPE>(z, z_block, z_tok, s, p, requests, longest, stream);                                        \
  }
PTL_GATED_LRU(_f32, float)
PTL_GATED_LRU(_bf16, __nv_bfloat16)

// A step in which every request brings one token: returns -2 where it does not take the sizes.
PTL_EXPORT int ptl_gated_lru_single_bf16(void* out, int out_ld, int column, const void* u, const void* w, int s, const float* gate_bias,
                                         const float* rate, const void* y, int y_ld, const float* y_bias, float* state,
                                         const int* tok_req, const int* positions, const int* state_slot, int tokens, int n,
                                         float scale, void* stream) {
  using namespace ptl;
  const LruArgs p = {out, u, y, gate_bias, rate, y_bias, state, nullptr, positions, state_slot, n, out_ld, column, y_ld, scale};
  if (int rc = lru_check(p, s)) return rc;
  if (tokens > kLruSingleTokens || s % 8 != 0 || n % 8 != 0 || !aligned16(u) || !aligned16(w)) return -2;
  if (tokens <= 0) return 0;
  return launch_kernel("gated_lru_single", gated_lru_single_kernel, dim3((n + 7) / 8), dim3(256), 0, as_stream(stream),
                       (const __nv_bfloat16*)w, s, tok_req, tokens, p);
}
