// Mixes of a token and the one before it, and the square of relu.
//
// token_shift, per token t and mix i:  out[i, t] = h[t] + (h' - h[t]) * mu[i], h' being the row before t of the same
// request: the neighbour in the step, or for a portion's first token the request's kept row, zeros at position 0.  The
// block of a portion's first token then keeps the portion's last row in the slot; no other block touches it.
//
// relu2, elementwise: max(z, 0)^2.
#include "common.cuh"

namespace ptl {

constexpr int kShiftMixes = 8;     // mixes at most

// A thread takes one packet of V elements of one token and all mixes (V 1: single elements).
template <typename T, int V>
__global__ void __launch_bounds__(256)
token_shift_kernel(T* __restrict__ out, long long plane, const T* __restrict__ h, const float* __restrict__ mu, int mixes, int width,
                   float* __restrict__ last, const int* __restrict__ q_start, const int* __restrict__ tok_req,
                   const int* __restrict__ positions, const int* __restrict__ state_slot) {
  const int t = blockIdx.x;
  const int r = tok_req[t];               // inputs of the step
  pdl_wait();
  pdl_launch_dependents();
  if (r < 0 || state_slot[r] < 0) return;
  const int i = (blockIdx.y * 256 + threadIdx.x) * V;
  if (i >= width) return;
  const int lo = q_start[r];
  float cur[V], old[V];
  auto row = [&](const T* src, float* dst) {
    if constexpr (V == 1) {
      dst[0] = to_f32(*src);
    } else {
      const Vec16<T> v = load16(src);
#pragma unroll
      for (int e = 0; e < V; ++e) dst[e] = v.get(e);
    }
  };
  row(h + (size_t)t * width + i, cur);
  if (t > lo) {
    row(h + (size_t)(t - 1) * width + i, old);
  } else {
    float* kept = last + (size_t)state_slot[r] * width + i;
    const bool fresh = positions[t] == 0;
#pragma unroll
    for (int e = 0; e < V; ++e) old[e] = fresh ? 0.f : kept[e];
    float end[V];
    row(h + (size_t)(q_start[r + 1] - 1) * width + i, end);
#pragma unroll
    for (int e = 0; e < V; ++e) kept[e] = end[e];
  }
#pragma unroll
  for (int e = 0; e < V; ++e) old[e] -= cur[e];
  for (int m = 0; m < mixes; ++m) {
    T* dst = out + m * plane + (size_t)t * width + i;
    const float* mm = mu + (size_t)m * width + i;
    if constexpr (V == 1) {
      *dst = from_f32<T>(fmaf(old[0], mm[0], cur[0]));
    } else {
      Vec16<T> v;
#pragma unroll
      for (int e = 0; e < V; e += 4) {
        const float4 c = *reinterpret_cast<const float4*>(mm + e);
        v.set(e, fmaf(old[e], c.x, cur[e]));
        v.set(e + 1, fmaf(old[e + 1], c.y, cur[e + 1]));
        v.set(e + 2, fmaf(old[e + 2], c.z, cur[e + 2]));
        v.set(e + 3, fmaf(old[e + 3], c.w, cur[e + 3]));
      }
      store16(dst, v);
    }
  }
}

template <typename T>
int token_shift(void* out, long long plane, const void* h, const float* mu, int mixes, int tokens, int width, float* last,
                const int* q_start, const int* tok_req, const int* positions, const int* state_slot, void* stream) {
  PTL_REQUIRE(tokens >= 0 && width > 0 && mixes >= 1 && mixes <= kShiftMixes && plane >= (long long)tokens * width,
              "token_shift: bad sizes tokens=%d width=%d mixes=%d", tokens, width, mixes);
  if (tokens == 0) return 0;
  constexpr int VN = Vec16<T>::N;
  if (width % VN == 0 && plane % VN == 0 && aligned16(out) && aligned16(h) && aligned16(mu) && width % 4 == 0)
    return launch_kernel("token_shift", token_shift_kernel<T, VN>, dim3(tokens, (width + 256 * VN - 1) / (256 * VN)), dim3(256), 0,
                         as_stream(stream), (T*)out, plane, (const T*)h, mu, mixes, width, last, q_start, tok_req, positions, state_slot);
  return launch_kernel("token_shift", token_shift_kernel<T, 1>, dim3(tokens, (width + 255) / 256), dim3(256), 0, as_stream(stream), (T*)out,
                       plane, (const T*)h, mu, mixes, width, last, q_start, tok_req, positions, state_slot);
}

// A thread takes one packet of 16 bytes; the elements after the last whole packet go one by one.
template <typename T>
__global__ void __launch_bounds__(256) relu2_kernel(T* __restrict__ x, long long n, long long packets) {
  constexpr int PER = Vec16<T>::N;
  pdl_wait();
  pdl_launch_dependents();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < packets) {
    Vec16<T> v = load16(x + i * PER);
#pragma unroll
    for (int e = 0; e < PER; ++e) { const float z = fmaxf(v.get(e), 0.f); v.set(e, z * z); }
    store16(x + i * PER, v);
  } else {
    const long long j = packets * PER + (i - packets);
    if (j < n) { const float z = fmaxf(to_f32(x[j]), 0.f); x[j] = from_f32<T>(z * z); }
  }
}

template <typename T>
int relu2(void* x, long long n, void* stream) {
  PTL_REQUIRE(n >= 0, "relu2: bad size");
  if (n == 0) return 0;
  const long long packets = aligned16(x) ? n / Vec16<T>::N : 0;
  const long long threads = packets + (n - packets * Vec16<T>::N);
  return launch_kernel("relu2", relu2_kernel<T>, dim3((unsigned)((threads + 255) / 256)), dim3(256), 0, as_stream(stream), (T*)x, n, packets);
}

}  // namespace ptl

#define PTL_TOKEN_SHIFT(SUFFIX, TYPE)                                                                                             \
  PTL_EXPORT int ptl_token_shift##SUFFIX(void* out, long long plane, const void* h, const float* mu, int mixes, int tokens,        \
                                         int width, float* last, const int* q_start, const int* tok_req, const int* positions,    \
                                         const int* state_slot, void* stream) {                                                   \
    return ptl::token_shift<TYPE>(out, plane, h, mu, mixes, tokens, width, last, q_start, tok_req, positions, state_slot, stream); \
  }                                                                                                                               \
  PTL_EXPORT int ptl_relu2##SUFFIX(void* x, long long n, void* stream) { return ptl::relu2<TYPE>(x, n, stream); }
PTL_TOKEN_SHIFT(_f32, float)
PTL_TOKEN_SHIFT(_bf16, __nv_bfloat16)
