// Linear-attention walks: per head a float32 state S [d, dv] that decays and takes up k_t v_t^T token by token.  Forms:
//
//   sigmoid  S <- diag(a_t) S + k_t v_t^T,  o_t = S^T q_t,  a_t = sigmoid(z_t + b)^(1/tau) = exp(logsigmoid(z_t + b) / tau)
//   fixed    the same with one fixed decay per head (retention)
//   bonus    o_t = (S + diag(u) k_t v_t^T)^T q_t, then S <- diag(a_t) S + k_t v_t^T, the decays a_t given (RWKV)
//   step     S <- exp(-rate_h s_t) S + s_t k_t v_t^T, o_t = S^T q_t + D_h v_t, s_t = softplus(dt_t + dt_bias_h) per head and
//            token (state space), q and k shared by groups of heads
//
// q_scale and k_scale multiply queries and keys.  q, k and v are rows of T elements with a pitch each; head h's q and k start
// at (h / per_qk) * d, its v at h * dv.  z is float32 [T, H*d], before the bias or the decay itself, dt float32 [T, H].
// A block owns COLS (32 or 16) columns of one head's state for one request and walks the request's
// tokens of this step in order.  Neighbouring threads are neighbouring columns; each of the 256 / COLS groups of them holds
// every eighth (sixteenth) packet of four of the d rows in registers (as pairs: the products and sums are the two-wide float32
// instructions, which round each half like the scalar forms), so the q, k and decay values a warp needs
// are the same for all its lanes (for each half of them): one shared-memory wavefront per packet.  16 columns are taken
// where blocks of 32 would leave half the SMs empty (measured at 2,048 tokens of one request: 64 blocks of 32 columns 358 us, 128 of
// 16 274 us; from about a block per SM on, staging every token twice as often costs more than it brings).  (With 8 lanes per column
// and the rows spread over the lanes the kernel was bound by shared-memory bandwidth, 437 wavefronts a
// token.)  Nothing in the walk waits on a shuffle; the groups' partial read-outs of a batch meet in
// shared memory.  Tokens come through shared memory in batches (q scaled, decay worked out while
// staging; the next batch's values are requested before the walk over this one).  What a token adds to its own read-out
// beside S (the bonus's sum over q u k, or D) is one number per token and head times v, added where the parts meet.  The state of a
// request is read from its slot unless the portion starts at position 0 and written back at the end.
// Everything after the loads is float32; a state does not depend on how the request was cut into steps or on what else the
// step holds, a read-out only through the grouping of its sum (16 or 32 columns).
#include "common.cuh"

namespace ptl {

constexpr int kGlaThreads = 256;
constexpr int kGlaNarrowBlocks = 74;      // up to so many blocks of 32 columns (half the SMs), blocks take 16

enum GlaForm { kGlaSigmoid = 0, kGlaFixed = 1, kGlaBonus = 2, kGlaStep = 3 };

struct GlaArgs {
  float* out;                     // [T, H*dv]
  const void *q, *k, *v;
  int q_ld, k_ld, v_ld, per_qk;
  const float *z, *bias;          // sigmoid; bonus: z is the decay, no bias
  float inv_tau;                  // sigmoid
  const float* head;              // fixed: the decay; step: the rate
  const float *dt, *dt_bias;      // step
  const float* extra;             // bonus: u [H*d]; step: D [H]
  float* state;
  const int *q_start, *positions, *state_slot;
  int H, d, dv;
  float q_scale, k_scale;
};

__device__ __forceinline__ float log_sigmoid_f32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float gla_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

template <typename T, int COLS, int RPL, int TB, int FORM>   // RPL rows per thread (d <= 256 / COLS * RPL), TB tokens per batch
__global__ void __launch_bounds__(kGlaThreads)
gla_scan_kernel(const GlaArgs p) {
  constexpr int kGroups = kGlaThreads / COLS;      // threads per column
  constexpr int DP = kGroups * RPL;
  constexpr bool kChannel = FORM == kGlaSigmoid || FORM == kGlaBonus;      // a decay per channel
  __shared__ __align__(16) float s_q[TB][DP], s_k[TB][DP], s_a[kChannel ? TB : 1][kChannel ? DP : 4];
  __shared__ float s_v[TB][COLS];
  __shared__ float s_part[TB][kGroups][COLS];              // a group's part of a token's read-out, per column
  __shared__ float s_step[2][TB], s_dec[2][TB];            // step form: a token's step size and decay, this batch's and the next's
  __shared__ float s_own[TB];                              // bonus form: sum of q u k
  pdl_wait();
  pdl_launch_dependents();
  const int r = blockIdx.z, h = blockIdx.y;
  const int t0 = p.q_start[r], t1 = p.q_start[r + 1];
  const int slot = p.state_slot[r];
  if (t1 <= t0 || slot < 0) return;
  const int H = p.H, d = p.d, dv = p.dv;
  const int tid = threadIdx.x;
  const int col = tid % COLS, grp = tid / COLS;            // grp: which share of the rows
  const int lane = tid & 31, warp = tid >> 5;
  const int e = blockIdx.x * COLS + col;
  const bool live = e < dv;
  // rows of this thread: packets of four, its packet m being packet m * kGroups + grp of the column
  auto row_of = [&](int i) { return ((i >> 2) * kGroups + grp) * 4 + (i & 3); };
  float* st = p.state + (((size_t)slot * H + h) * d) * dv;
  float2 S[RPL / 2];
  const bool fresh = p.positions[t0] == 0;
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const float s = (!fresh && live && row_of(i) < d) ? st[(size_t)row_of(i) * dv + e] : 0.f;
    if (i & 1) S[i >> 1].y = s; else S[i >> 1].x = s;
  }
  const T* qp = reinterpret_cast<const T*>(p.q) + (size_t)(h / p.per_qk) * d;
  const T* kp = reinterpret_cast<const T*>(p.k) + (size_t)(h / p.per_qk) * d;
  const T* vp = reinterpret_cast<const T*>(p.v) + (size_t)h * dv + blockIdx.x * COLS;
  const int vcols = min(COLS, dv - blockIdx.x * COLS);

  // A thread fetches the same column c of q, k and z for tokens j0, j0 + step, ...: the next batch's values are
  // requested before the walk over this batch and kept as fetched; they are converted (and the decay worked out)
  // when they go to shared memory, after the walk.
  constexpr int NE = TB * DP / kGlaThreads, NV = (TB * COLS + kGlaThreads - 1) / kGlaThreads;
  constexpr int kTokStep = kGlaThreads / DP > 0 ? kGlaThreads / DP : 1;
  static_assert(kGlaThreads % DP == 0 && NE * kTokStep == TB, "a thread's column must not change between its turns");
  const int c_mine = tid % DP, j_mine = tid / DP;
  const float b_mine = (FORM == kGlaSigmoid && c_mine < d) ? p.bias[h * d + c_mine] : 0.f;
  const float head_h = kChannel ? 0.f : p.head[h];         // the fixed decay, or the step form's rate
  const float dt_bias = FORM == kGlaStep ? p.dt_bias[h] : 0.f, skip = FORM == kGlaStep ? p.extra[h] : 0.f;
  float bonus[(DP + 31) / 32];
  if constexpr (FORM == kGlaBonus) {
#pragma unroll
    for (int i = 0; i < (DP + 31) / 32; ++i) bonus[i] = lane + 32 * i < d ? p.extra[h * d + lane + 32 * i] : 0.f;
  }
  T rq[NE], rk[NE], rv[NV];
  float rz[NE], rdt = 0.f;
  auto fetch = [&](int tb) {
    const int nt = min(TB, t1 - tb);
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      const int j = j_mine + i * kTokStep;
      const bool ok = j < nt && c_mine < d;
      const size_t t = (size_t)(tb + (ok ? j : 0));
      rq[i] = ok ? qp[t * p.q_ld + c_mine] : from_f32<T>(0.f);
      rk[i] = ok ? kp[t * p.k_ld + c_mine] : from_f32<T>(0.f);
      if constexpr (kChannel) rz[i] = ok ? p.z[t * H * d + h * d + c_mine] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int idx = tid + i * kGlaThreads;
      const int j = idx / COLS, c = idx % COLS;
      rv[i] = (j < nt && c < vcols) ? vp[(size_t)(tb + j) * p.v_ld + c] : from_f32<T>(0.f);
    }
    if (FORM == kGlaStep && tid < nt) rdt = p.dt[(size_t)(tb + tid) * H + h];
  };
  auto stage = [&](int buf) {
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      const int j = j_mine + i * kTokStep;
      s_q[j][c_mine] = to_f32(rq[i]) * p.q_scale;
      float k = to_f32(rk[i]) * p.k_scale;
      if constexpr (FORM == kGlaStep) k *= s_step[buf][j];
      s_k[j][c_mine] = k;
      if constexpr (FORM == kGlaSigmoid) s_a[j][c_mine] = c_mine < d ? expf(log_sigmoid_f32(rz[i] + b_mine) * p.inv_tau) : 0.f;
      if constexpr (FORM == kGlaBonus) s_a[j][c_mine] = rz[i];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int idx = tid + i * kGlaThreads;
      if (idx < TB * COLS) s_v[idx / COLS][idx % COLS] = to_f32(rv[i]);
    }
  };
  fetch(t0);
  int buf = 0;
  for (int tb = t0; tb < t1; tb += TB, buf ^= 1) {
    const int nt = min(TB, t1 - tb);
    if (FORM == kGlaStep && tid < TB) {    // (the walk over the batch before reads the other buffer)
      const float s = tid < nt ? gla_softplus(rdt + dt_bias) : 0.f;
      s_step[buf][tid] = s;
      s_dec[buf][tid] = decay_exp(-head_h * s);
    }
    __syncthreads();                       // the walk over the batch before is done with the staged tokens
    stage(buf);
    __syncthreads();
    if (tb + TB < t1) fetch(tb + TB);
    if constexpr (FORM == kGlaBonus) {     // read where the parts meet, behind the walk's barrier
      for (int j = warp; j < nt; j += kGlaThreads / 32) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < (DP + 31) / 32; ++i) s = fmaf(s_q[j][lane + 32 * i] * s_k[j][lane + 32 * i], bonus[i], s);
        s = warp_sum(s);
        if (lane == 0) s_own[j] = s;
      }
    }
    auto token = [&](int j) {
      const float v = s_v[j][col];
      const float2 v2 = make_float2(v, v);
      float2 dec = make_float2(head_h, head_h);
      if constexpr (FORM == kGlaStep) dec.x = dec.y = s_dec[buf][j];
      float2 acc0 = make_float2(0.f, 0.f), acc1 = make_float2(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < RPL; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(&s_k[j][row_of(i)]);
        const float4 q4 = *reinterpret_cast<const float4*>(&s_q[j][row_of(i)]);
        float2 a0 = dec, a1 = dec;
        if constexpr (kChannel) {
          const float4 a4 = *reinterpret_cast<const float4*>(&s_a[j][row_of(i)]);
          a0 = make_float2(a4.x, a4.y);
          a1 = make_float2(a4.z, a4.w);
        }
        const float2 q0 = make_float2(q4.x, q4.y), q1 = make_float2(q4.z, q4.w);
        float2& S0 = S[i >> 1];
        float2& S1 = S[(i >> 1) + 1];
        if constexpr (FORM == kGlaBonus) {          // the read-out sees the state as it was
          acc0 = __ffma2_rn(q0, S0, acc0);
          acc1 = __ffma2_rn(q1, S1, acc1);
        }
        S0 = __ffma2_rn(a0, S0, __fmul2_rn(make_float2(k4.x, k4.y), v2));
        S1 = __ffma2_rn(a1, S1, __fmul2_rn(make_float2(k4.z, k4.w), v2));
        if constexpr (FORM != kGlaBonus) {
          acc0 = __ffma2_rn(q0, S0, acc0);
          acc1 = __ffma2_rn(q1, S1, acc1);
        }
      }
      s_part[j][grp][col] = (acc0.x + acc0.y) + (acc1.x + acc1.y);
    };
    if (nt == TB) {
#pragma unroll 4
      for (int j = 0; j < TB; ++j) token(j);            // (unrolled: the next token's loads and products start under this one's sums)
    } else {
      for (int j = 0; j < nt; ++j) token(j);
    }
    __syncthreads();
    // the groups' parts of every read-out of the batch, added in the order of the groups
    for (int idx = tid; idx < nt * COLS; idx += kGlaThreads) {
      const int j = idx / COLS, c = idx % COLS;
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < kGroups; ++w) sum += s_part[j][w][c];
      if constexpr (FORM == kGlaBonus) sum = fmaf(s_own[j], s_v[j][c], sum);
      if constexpr (FORM == kGlaStep) sum = fmaf(skip, s_v[j][c], sum);
      if (c < vcols) p.out[(size_t)(tb + j) * H * dv + (size_t)h * dv + blockIdx.x * COLS + c] = sum;
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < RPL; ++i)
      if (row_of(i) < d) st[(size_t)row_of(i) * dv + e] = (i & 1) ? S[i >> 1].y : S[i >> 1].x;
  }
}

template <typename T, int FORM>
int gla_launch(const char* what, const GlaArgs& p, int requests, void* stream) {
  PTL_REQUIRE(requests >= 0 && p.H > 0 && p.d > 0 && p.dv > 0 && p.per_qk > 0 && p.H % p.per_qk == 0, "%s: bad sizes", what);
  PTL_REQUIRE(p.d <= 256, "%s: head size %d, at most 256", what, p.d);
  PTL_REQUIRE(p.q_ld >= p.H / p.per_qk * p.d && p.k_ld >= p.H / p.per_qk * p.d && p.v_ld >= p.H * p.dv, "%s: rows are too short", what);
  PTL_REQUIRE(p.H <= 65535 && requests <= 65535, "%s: too many heads or requests", what);
  if (requests == 0) return 0;
#define PTL_GLA_LAUNCH(COLS, RPL, TB)                                                                                        \
  return launch_kernel(what, gla_scan_kernel<T, COLS, RPL, TB, FORM>, dim3((p.dv + COLS - 1) / COLS, p.H, requests),           \
                       dim3(kGlaThreads), 0, as_stream(stream), p)
  if (p.d <= 32) PTL_GLA_LAUNCH(32, 4, 16);
  const bool narrow = (long long)((p.dv + 31) / 32) * p.H * requests <= kGlaNarrowBlocks;
  if (p.d <= 64) { if (narrow) PTL_GLA_LAUNCH(16, 4, 16); PTL_GLA_LAUNCH(32, 8, 16); }
  if (p.d <= 128) { if (narrow) PTL_GLA_LAUNCH(16, 8, 16); PTL_GLA_LAUNCH(32, 16, 16); }
  PTL_GLA_LAUNCH(32, 32, 8);
#undef PTL_GLA_LAUNCH
}

template <typename T>
int gla_scan(float* out, const void* proj, int ld, const float* z, const float* bias, float inv_tau, float* state,
             const int* q_start, const int* positions, const int* state_slot, int requests, int H, int d, int dv,
             float q_scale, const float* head_decay, float k_scale, void* stream) {
  PTL_REQUIRE((z && bias) || head_decay, "gla_scan: neither a decay per channel nor one per head");
  PTL_REQUIRE(ld >= 2 * H * d + H * dv, "gla_scan: rows of %d elements are too short", ld);
  const T* rows = (const T*)proj;
  GlaArgs p{};
  p.out = out; p.q = rows; p.k = rows + (size_t)H * d; p.v = rows + 2 * (size_t)H * d; p.q_ld = p.k_ld = p.v_ld = ld; p.per_qk = 1;
  p.z = z; p.bias = bias; p.inv_tau = inv_tau; p.head = head_decay; p.state = state;
  p.q_start = q_start; p.positions = positions; p.state_slot = state_slot; p.H = H; p.d = d; p.dv = dv; p.q_scale = q_scale; p.k_scale = k_scale;
  if (z) return gla_launch<T, kGlaSigmoid>("gla_scan", p, requests, stream);
  return gla_launch<T, kGlaFixed>("gla_scan", p, requests, stream);
}

// rkv: the rows of r, k and v are `plane` elements apart, each [T, H*d].
template <typename T>
int wkv_scan(float* out, const void* rkv, long long plane, const float* decay, const float* u, float* state,
             const int* q_start, const int* positions, const int* state_slot, int requests, int H, int d, void* stream) {
  PTL_REQUIRE(decay && u && plane >= 0, "wkv_scan: missing operands");
  const T* rows = (const T*)rkv;
  GlaArgs p{};
  p.out = out; p.q = rows; p.k = rows + plane; p.v = rows + 2 * plane; p.q_ld = p.k_ld = p.v_ld = H * d; p.per_qk = 1;
  p.z = decay; p.extra = u; p.state = state;
  p.q_start = q_start; p.positions = positions; p.state_slot = state_slot; p.H = H; p.d = d; p.dv = d; p.q_scale = p.k_scale = 1.f;
  return gla_launch<T, kGlaBonus>("wkv_scan", p, requests, stream);
}

// xbc rows: [x: H * dv | B: G * n | C: G * n].
template <typename T>
int state_space_scan(float* out, const void* xbc, int ld, const float* dt, const float* dt_bias, const float* rate, const float* D,
                     float* state, const int* q_start, const int* positions, const int* state_slot, int requests, int H, int G, int n,
                     int dv, void* stream) {
  PTL_REQUIRE(dt && dt_bias && rate && D && G > 0 && H % G == 0, "state_space_scan: bad arguments");
  PTL_REQUIRE(ld >= H * dv + 2 * G * n, "state_space_scan: rows of %d elements are too short", ld);
  const T* rows = (const T*)xbc;
  GlaArgs p{};
  p.out = out; p.v = rows; p.k = rows + (size_t)H * dv; p.q = rows + (size_t)H * dv + (size_t)G * n; p.q_ld = p.k_ld = p.v_ld = ld;
  p.per_qk = H / G; p.dt = dt; p.dt_bias = dt_bias; p.head = rate; p.extra = D; p.state = state;
  p.q_start = q_start; p.positions = positions; p.state_slot = state_slot; p.H = H; p.d = n; p.dv = dv; p.q_scale = p.k_scale = 1.f;
  return gla_launch<T, kGlaStep>("state_space_scan", p, requests, stream);
}

}  // namespace ptl

#define PTL_GLA(SUFFIX, TYPE)                                                                                                   \
  PTL_EXPORT int ptl_gla_scan##SUFFIX(float* out, const void* proj, int ld, const float* z, const float* bias, float inv_tau,    \
                                      float* state, const int* q_start, const int* positions, const int* state_slot,            \
                                      int requests, int H, int d, int dv, float q_scale, const float* head_decay,               \
                                      float k_scale, void* stream) {                                                            \
    return ptl::gla_scan<TYPE>(out, proj, ld, z, bias, inv_tau, state, q_start, positions, state_slot, requests, H, d, dv,       \
                               q_scale, head_decay, k_scale, stream);                                                           \
  }                                                                                                                             \
  PTL_EXPORT int ptl_wkv_scan##SUFFIX(float* out, const void* rkv, long long plane, const float* decay, const float* u,          \
                                      float* state, const int* q_start, const int* positions,                   \
                                      const int* state_slot, int requests, int H, int d, void* stream) {                        \
    return ptl::wkv_scan<TYPE>(out, rkv, plane, decay, u, state, q_start, positions, state_slot, requests, H, d, stream);      \
  }                                                                                                                             \
  PTL_EXPORT int ptl_state_space_scan##SUFFIX(float* out, const void* xbc, int ld, const float* dt, const float* dt_bias,        \
                                              const float* rate, const float* D, float* state, const int* q_start,              \
                                              const int* positions, const int* state_slot, int requests, int H, int G, int n,   \
                                              int dv, void* stream) {                                                           \
    return ptl::state_space_scan<TYPE>(out, xbc, ld, dt, dt_bias, rate, D, state, q_start, positions, state_slot, requests, H, G, \
                                       n, dv, stream);                                                                          \
  }
PTL_GLA(_f32, float)
PTL_GLA(_bf16, __nv_bfloat16)
