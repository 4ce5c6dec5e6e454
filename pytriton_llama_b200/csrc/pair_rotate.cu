// Rotation of neighbouring pairs with the cache write, for keys that are also the values.
//
// pair_angles, per token and pair i < half: (cos, sin) of position * freq[i], the angle in 64 bits, times `amplitude`,
// as float32; made once per step and frequency table and read by every layer.
//
// pair_rotate_store, per token of the step, on the projection's output [T, q | k (| v)], with `bias` [q | k (| v)] added
// in float32 to all of it:
//   entries 2i and 2i + 1, i < dims/2, of every q and k head are turned by the token's angles;
//   q is written back in place, k goes to the token's slot of the cache and nowhere else;
//   the value that goes beside it is v, or with `values_are_keys` (no v in the projection) k before it is turned.
// A page of the cache holds its keys, then its values, as the attention kernels read it.
#include "common.cuh"

namespace ptl {

__global__ void __launch_bounds__(128)
pair_angles_kernel(float2* __restrict__ table, const int* __restrict__ positions, const double* __restrict__ freq, int n, int half,
                   float amplitude) {
  pdl_wait();
  pdl_launch_dependents();
  const int idx = blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= n) return;
  double s, c;
  sincos((double)positions[idx / half] * freq[idx % half], &s, &c);
  table[idx] = make_float2((float)c * amplitude, (float)s * amplitude);
}

template <typename T>
__global__ void __launch_bounds__(256)
pair_rotate_store_kernel(T* __restrict__ proj, int ld, int H, int G, int d, int dv, const float* __restrict__ bias,
                         const float2* __restrict__ table, int dims, int values_are_keys, const int* __restrict__ slots,
                         T* __restrict__ cache, int page_size, long long num_slots, int vec_ok) {
  const int t = blockIdx.x;
  long long slot = (slots && cache) ? (long long)slots[t] : -1;      // an input of the step
  if (slot >= num_slots) slot = -1;
  pdl_wait();
  pdl_launch_dependents();
  T* row = proj + (size_t)t * ld;
  const int half = dims / 2;
  const float2* cs = table + (size_t)t * half;
  const int nq = H * d, nqk = (H + G) * d;
  T* kdst = nullptr;
  T* vdst = nullptr;
  if (slot >= 0) {
    const size_t page_stride = (size_t)G * page_size * (d + dv);
    const size_t page = (size_t)(slot / page_size), off = (size_t)(slot % page_size);
    kdst = cache + page * page_stride + off * d;                                  // + g * page_size * d
    vdst = cache + page * page_stride + (size_t)G * page_size * d + off * dv;     // + g * page_size * dv
  }
  constexpr int VN = Vec16<T>::N;
  if (vec_ok) {
    for (int i = threadIdx.x * VN; i < nqk; i += blockDim.x * VN) {
      const bool is_k = i >= nq;
      if (is_k && slot < 0) break;                        // nothing is kept of this token
      const int within = (is_k ? i - nq : i) % d;         // first entry of the packet within its head
      Vec16<T> v = load16(row + i);
      float x[VN];
#pragma unroll
      for (int e = 0; e < VN; ++e) x[e] = v.get(e);
      if (bias) {
#pragma unroll
        for (int e = 0; e < VN; e += 4) {
          const float4 b = __ldg(reinterpret_cast<const float4*>(bias + i + e));
          x[e] += b.x; x[e + 1] += b.y; x[e + 2] += b.z; x[e + 3] += b.w;
        }
      }
      const int g = is_k ? (i - nq) / d : 0;
      if (is_k && values_are_keys) {
#pragma unroll
        for (int e = 0; e < VN; ++e) v.set(e, x[e]);
        store16(vdst + (size_t)g * page_size * dv + within, v);
      }
      if (within < dims) {
#pragma unroll
        for (int e = 0; e < VN; e += 2) {
          if (within + e + 1 < dims) {
            const float2 a = cs[(within + e) >> 1];
            float o1, o2;
            rope_rotate(x[e], x[e + 1], a.x, a.y, o1, o2);
            x[e] = o1;
            x[e + 1] = o2;
          }
        }
      }
#pragma unroll
      for (int e = 0; e < VN; ++e) v.set(e, x[e]);
      if (is_k) store16(kdst + (size_t)g * page_size * d + within, v);
      else store16(row + i, v);
    }
  } else {
    const int per_head = (d + 1) / 2;                     // two neighbours per turn; an odd last entry alone
    for (int idx = threadIdx.x; idx < (H + G) * per_head; idx += blockDim.x) {
      const int h = idx / per_head, i = idx % per_head;
      const int e0 = 2 * i, e1 = 2 * i + 1;
      const bool is_k = h >= H;
      if (is_k && slot < 0) break;
      const size_t at = (size_t)h * d + e0;
      float a = to_f32(row[at]) + (bias ? bias[at] : 0.f);
      float b = e1 < d ? to_f32(row[at + 1]) + (bias ? bias[at + 1] : 0.f) : 0.f;
      if (is_k && values_are_keys) {
        T* vd = vdst + (size_t)(h - H) * page_size * dv;
        vd[e0] = from_f32<T>(a);
        if (e1 < d) vd[e1] = from_f32<T>(b);
      }
      if (e1 < dims) {
        const float2 c = cs[i];
        float o1, o2;
        rope_rotate(a, b, c.x, c.y, o1, o2);
        a = o1;
        b = o2;
      }
      T* dst = is_k ? kdst + (size_t)(h - H) * page_size * d : row + (size_t)h * d;
      dst[e0] = from_f32<T>(a);
      if (e1 < d) dst[e1] = from_f32<T>(b);
    }
  }
  if (vdst && !values_are_keys) {
    for (int i = threadIdx.x; i < G * dv; i += blockDim.x) {
      const int g = i / dv, e = i % dv;
      vdst[(size_t)g * page_size * dv + e] = from_f32<T>(to_f32(row[nqk + i]) + (bias ? bias[nqk + i] : 0.f));
    }
  }
}

template <typename T>
int pair_rotate_store(void* proj, int tokens, int ld, int H, int G, int d, int dv, const float* bias, const void* table, int dims,
                      int values_are_keys, const int* slots, void* cache, int page_size, long long num_slots, void* stream) {
  PTL_REQUIRE(tokens >= 0 && H > 0 && G >= 0 && d > 0 && dv > 0 && page_size > 0, "pair_rotate_store: bad sizes");
  PTL_REQUIRE(!values_are_keys || dv == d, "pair_rotate_store: values of %d entries that are keys of %d", dv, d);
  PTL_REQUIRE(ld >= (H + G) * d + (values_are_keys ? 0 : G * dv), "pair_rotate_store: rows of %d elements are too short", ld);
  PTL_REQUIRE(dims >= 0 && dims % 2 == 0 && dims <= d && (dims == 0 || table), "pair_rotate_store: rotary width %d of head size %d", dims, d);
  if (tokens == 0) return 0;
  constexpr int VN = Vec16<T>::N;
  const int vec_ok = d % VN == 0 && dv % VN == 0 && ld % VN == 0 && aligned16(proj) && (!cache || aligned16(cache)) &&
                     (!bias || aligned16(bias));
  return launch_kernel("pair_rotate_store", pair_rotate_store_kernel<T>, dim3(tokens), dim3(256), 0, as_stream(stream), (T*)proj, ld, H,
                       G, d, dv, bias, (const float2*)table, dims, values_are_keys, slots, (T*)cache, page_size, num_slots, vec_ok);
}

}  // namespace ptl

PTL_EXPORT int ptl_pair_angles(void* table, const int* positions, const double* freq, int tokens, int half, float amplitude, void* stream) {
  PTL_REQUIRE(tokens >= 0 && half > 0 && (long long)tokens * half < (1ll << 31), "pair_angles: bad sizes tokens=%d pairs=%d", tokens, half);
  if (tokens == 0) return 0;
  const int n = tokens * half;
  return ptl::launch_kernel("pair_angles", ptl::pair_angles_kernel, dim3((n + 127) / 128), dim3(128), 0, ptl::as_stream(stream),
                            (float2*)table, positions, freq, n, half, amplitude);
}

#define PTL_PAIR_ROTATE(SUFFIX, TYPE)                                                                                              \
  PTL_EXPORT int ptl_pair_rotate_store##SUFFIX(void* proj, int tokens, int ld, int H, int G, int d, int dv, const float* bias,      \
                                               const void* table, int dims, int values_are_keys, const int* slots, void* cache,    \
                                               int page_size, long long num_slots, void* stream) {                                 \
    return ptl::pair_rotate_store<TYPE>(proj, tokens, ld, H, G, d, dv, bias, table, dims, values_are_keys, slots, cache,           \
                                        page_size, num_slots, stream);                                                             \
  }
PTL_PAIR_ROTATE(_f32, float)
PTL_PAIR_ROTATE(_bf16, __nv_bfloat16)
