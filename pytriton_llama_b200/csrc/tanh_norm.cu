// A norm without statistics, y = tanh(alpha * s) * w + b entry by entry, fused with what comes before it: a sub-layer's
// output, in one of three forms, times a vector, added into the float32 residual.  Per row m (r = rows ? rows[m] : m):
//
//   o = x[r]                                                          (x of T or float32; or nothing)
//   o = shared[r] + sum_k weights[r, k] * C[pos[r, k]]                (experts: in the order of the choices)
//   o = (1 / members) sum_m a_m[r] * rsqrt(mean(a_m[r]^2) + eps) * w_m   (members 1 or 2)
//   s = residual_in[r] + scale * o;   residual_out[m] = s (when given);   y[m] = tanh(alpha * s) * w + b
//
// float32 throughout; y is rounded once.  The first two forms have no sum over the row: a thread takes four neighbours
// and waits for nobody.  The third takes one block per row.
#include "common.cuh"

namespace ptl {

struct TanhNormArgs {
  void* y;
  float* residual_out;
  const float* residual_in;
  const float *scale, *w, *b;
  float alpha;
  const int* rows;
  int width;
  // experts
  const float *C, *weights;
  const int* pos;
  int top;
};

template <typename A>
__device__ __forceinline__ float4 tn_load4(const A* p) {
  if constexpr (sizeof(A) == 4) {
    return *reinterpret_cast<const float4*>(p);
  } else {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
  }
}
template <typename T>
__device__ __forceinline__ void tn_store4(T* p, float4 v) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = v;
  } else {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = raw;
  }
}
__device__ __forceinline__ float tn_norm(float s, float alpha, float w, float b) { return fmaf(tanhf(alpha * s), w, b); }

// The sum and the norm of four neighbours whose output is `o`.
template <typename T>
__device__ __forceinline__ void tn_finish4(const TanhNormArgs& p, int m, int i, float4 o, bool have, float4 res) {
  float4 s = res;
  if (have) {
    if (p.scale) {
      const float4 c = *reinterpret_cast<const float4*>(p.scale + i);
      s = make_float4(fmaf(c.x, o.x, s.x), fmaf(c.y, o.y, s.y), fmaf(c.z, o.z, s.z), fmaf(c.w, o.w, s.w));
    } else {
      s = make_float4(s.x + o.x, s.y + o.y, s.z + o.z, s.w + o.w);
    }
  }
  if (p.residual_out && (have || p.residual_out != p.residual_in)) *reinterpret_cast<float4*>(p.residual_out + (size_t)m * p.width + i) = s;
  const float4 w = *reinterpret_cast<const float4*>(p.w + i), b = *reinterpret_cast<const float4*>(p.b + i);
  tn_store4<T>((T*)p.y + (size_t)m * p.width + i,
               make_float4(tn_norm(s.x, p.alpha, w.x, b.x), tn_norm(s.y, p.alpha, w.y, b.y), tn_norm(s.z, p.alpha, w.z, b.z),
                           tn_norm(s.w, p.alpha, w.w, b.w)));
}
template <typename T>
__device__ __forceinline__ void tn_finish(const TanhNormArgs& p, int m, int r, int i, float o, bool have) {
  float s = p.residual_in ? p.residual_in[(size_t)r * p.width + i] : 0.f;
  if (have) s = p.scale ? fmaf(p.scale[i], o, s) : s + o;
  if (p.residual_out && (have || p.residual_out != p.residual_in)) p.residual_out[(size_t)m * p.width + i] = s;
  ((T*)p.y)[(size_t)m * p.width + i] = from_f32<T>(tn_norm(s, p.alpha, p.w[i], p.b[i]));
}

// x: the output (or null), or with C the shared expert's (or null).
template <typename T, typename A>
__global__ void __launch_bounds__(256)
add_tanh_norm_kernel(const A* __restrict__ x, const TanhNormArgs p, int vec_ok) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, r = p.rows ? p.rows[m] : m;
  const bool have = x || p.C;
  if (vec_ok) {
    const int i = (blockIdx.y * 256 + threadIdx.x) * 4;
    if (i >= p.width) return;
    float4 res = p.residual_in ? *reinterpret_cast<const float4*>(p.residual_in + (size_t)r * p.width + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    float4 o = x ? tn_load4<A>(x + (size_t)r * p.width + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    if (p.C) {
      for (int k0 = 0; k0 < p.top; k0 += 4) {        // four choices' rows are requested together, then added in order
        float4 v[4];
        float wk[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int row = k0 + u < p.top ? p.pos[(size_t)r * p.top + k0 + u] : -1;
          wk[u] = row < 0 ? 0.f : p.weights[(size_t)r * p.top + k0 + u];
          v[u] = row < 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(p.C + (size_t)row * p.width + i);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
          o = make_float4(fmaf(wk[u], v[u].x, o.x), fmaf(wk[u], v[u].y, o.y), fmaf(wk[u], v[u].z, o.z), fmaf(wk[u], v[u].w, o.w));
      }
    }
    tn_finish4<T>(p, m, i, o, have, res);
    return;
  }
  for (int i = blockIdx.y * 1024 + threadIdx.x; i < min(p.width, (int)(blockIdx.y + 1) * 1024); i += 256) {
    float o = x ? to_f32(x[(size_t)r * p.width + i]) : 0.f;
    if (p.C)
      for (int k = 0; k < p.top; ++k) {
        const int row = p.pos[(size_t)r * p.top + k];
        if (row >= 0) o = fmaf(p.weights[(size_t)r * p.top + k], p.C[(size_t)row * p.width + i], o);
      }
    tn_finish<T>(p, m, r, i, o, have);
  }
}

// The mean of one or two normed outputs; NP packets of four per thread, held in registers (NP 0: walked twice instead).
template <typename T, typename A, int NP>
__global__ void __launch_bounds__(256)
members_tanh_norm_kernel(const A* __restrict__ a0, const A* __restrict__ a1, const float* __restrict__ w0, const float* __restrict__ w1,
                         int members, float eps, const TanhNormArgs p) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, r = p.rows ? p.rows[m] : m;
  const size_t row = (size_t)r * p.width;
  const float inv_w = 1.0f / (float)p.width, share = 1.0f / (float)members;
  float q0 = 0.f, q1 = 0.f;
  constexpr int N = NP > 0 ? NP : 1;
  float4 u[N], v[N], res[N];
  if constexpr (NP > 0) {
#pragma unroll
    for (int n = 0; n < NP; ++n) {        // everything this row reads is requested before the first sum
      const int i = (n * 256 + threadIdx.x) * 4;
      u[n] = v[n] = res[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < p.width) {
        u[n] = tn_load4<A>(a0 + row + i);
        if (members > 1) v[n] = tn_load4<A>(a1 + row + i);
        if (p.residual_in) res[n] = *reinterpret_cast<const float4*>(p.residual_in + row + i);
      }
    }
#pragma unroll
    for (int n = 0; n < NP; ++n) {
      q0 += fmaf(u[n].x, u[n].x, fmaf(u[n].y, u[n].y, fmaf(u[n].z, u[n].z, u[n].w * u[n].w)));
      q1 += fmaf(v[n].x, v[n].x, fmaf(v[n].y, v[n].y, fmaf(v[n].z, v[n].z, v[n].w * v[n].w)));
    }
  } else {
    for (int i = threadIdx.x; i < p.width; i += 256) {
      const float x0 = to_f32(a0[row + i]), x1 = members > 1 ? to_f32(a1[row + i]) : 0.f;
      q0 = fmaf(x0, x0, q0);
      q1 = fmaf(x1, x1, q1);
    }
  }
  const float r0 = share / sqrtf(block_sum(q0, red) * inv_w + eps);
  const float r1 = members > 1 ? share / sqrtf(block_sum(q1, red) * inv_w + eps) : 0.f;
  if constexpr (NP > 0) {
#pragma unroll
    for (int n = 0; n < NP; ++n) {
      const int i = (n * 256 + threadIdx.x) * 4;
      if (i >= p.width) continue;
      const float4 wa = *reinterpret_cast<const float4*>(w0 + i);
      float4 o = make_float4(u[n].x * r0 * wa.x, u[n].y * r0 * wa.y, u[n].z * r0 * wa.z, u[n].w * r0 * wa.w);
      if (members > 1) {
        const float4 wb = *reinterpret_cast<const float4*>(w1 + i);
        o = make_float4(fmaf(v[n].x * r1, wb.x, o.x), fmaf(v[n].y * r1, wb.y, o.y), fmaf(v[n].z * r1, wb.z, o.z), fmaf(v[n].w * r1, wb.w, o.w));
      }
      tn_finish4<T>(p, m, i, o, true, res[n]);
    }
  } else {
    for (int i = threadIdx.x; i < p.width; i += 256) {
      float o = to_f32(a0[row + i]) * r0 * w0[i];
      if (members > 1) o = fmaf(to_f32(a1[row + i]) * r1, w1[i], o);
      tn_finish<T>(p, m, r, i, o, true);
    }
  }
}

template <typename T, typename A>
int add_tanh_norm(const void* x, const void* a1, const float* w0, const float* w1, int members, float eps, const TanhNormArgs& p,
                  int out_rows, void* stream) {
  PTL_REQUIRE(out_rows >= 0 && p.width > 0 && p.y && p.w && p.b, "add_tanh_norm: bad arguments");
  PTL_REQUIRE(members >= 0 && members <= 2 && (members < 1 || (x && w0 && eps > 0.f && !p.C)) && (members < 2 || (a1 && w1)),
              "add_tanh_norm: %d members (at most 2, each with its weight)", members);
  PTL_REQUIRE(!p.C || (p.pos && p.weights && p.top > 0), "add_tanh_norm: experts without rows or weights");
  PTL_REQUIRE(!p.rows || !p.residual_out, "add_tanh_norm: picked rows keep no sum");
  if (out_rows == 0) return 0;
  const int vec_ok = p.width % 4 == 0 && aligned16(x) && aligned16(a1) && aligned16(w0) && aligned16(w1) && aligned16(p.y) && aligned16(p.w) &&
                     aligned16(p.b) && aligned16(p.scale) && aligned16(p.residual_in) && aligned16(p.residual_out) && aligned16(p.C);
  if (members > 0) {
#define PTL_TN_MEMBERS(NP)                                                                                                     \
    return launch_kernel("members_tanh_norm", members_tanh_norm_kernel<T, A, NP>, dim3(out_rows), dim3(256), 0,                  \
                         as_stream(stream), (const A*)x, (const A*)a1, w0, w1, members, eps, p)
    if (!vec_ok || p.width > 8192) PTL_TN_MEMBERS(0);
    if (p.width <= 1024) PTL_TN_MEMBERS(1);
    if (p.width <= 2048) PTL_TN_MEMBERS(2);
    if (p.width <= 4096) PTL_TN_MEMBERS(4);
    PTL_TN_MEMBERS(8);
#undef PTL_TN_MEMBERS
  }
  return launch_kernel("add_tanh_norm", add_tanh_norm_kernel<T, A>, dim3(out_rows, (p.width + 1023) / 1024), dim3(256), 0,
                       as_stream(stream), (const A*)x, p, vec_ok);
}

}  // namespace ptl

// x_f32: the sub-layer's output is float32 whatever the compute type
#define PTL_TANH_NORM(SUFFIX, TYPE)                                                                                              \
  PTL_EXPORT int ptl_add_tanh_norm##SUFFIX(void* y, float* residual_out, const float* residual_in, const void* x, int x_f32,      \
                                           const float* scale, const float* w, const float* b, float alpha, const int* rows,     \
                                           int out_rows, int width, const void* a1, const float* w0, const float* w1, int members, \
                                           float eps, const float* C, const int* pos, const float* weights, int top,             \
                                           void* stream) {                                                                       \
    const ptl::TanhNormArgs p = {y, residual_out, residual_in, scale, w, b, alpha, rows, width, C, weights, pos, top};           \
    if (x_f32) return ptl::add_tanh_norm<TYPE, float>(x, a1, w0, w1, members, eps, p, out_rows, stream);                         \
    return ptl::add_tanh_norm<TYPE, TYPE>(x, a1, w0, w1, members, eps, p, out_rows, stream);                                     \
  }
PTL_TANH_NORM(_f32, float)
PTL_TANH_NORM(_bf16, __nv_bfloat16)
