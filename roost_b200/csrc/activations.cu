// Activation functions of feed-forwards that are not gated, and gates that scale whole heads.
//
// xielu:          y = a_pos z^2 + z / 2 for z > 0, y = a_neg (exp(z) - 1 - z) + z / 2 for z <= 0, on the 32-bit value, rounded once.
//                 Vector form: 16 bytes a thread where the pointers and the count allow.
// relu_squared:   y = max(z, 0)^2, likewise.
// head_gate_mul:  x[t, h, :] *= sigmoid(g[t, col + h]), one gate a token and head, in place.
#include "common.cuh"

namespace roost {

__device__ __forceinline__ float xielu_f(float z, float a_pos, float a_neg) {
  return z > 0.f ? fmaf(a_pos * z, z, 0.5f * z) : fmaf(a_neg, expm1f(z) - z, 0.5f * z);
}

template <typename T>
__global__ void xielu_kernel(const T* __restrict__ x, T* __restrict__ out, size_t n, float a_pos, float a_neg) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) out[i] = from_float<T>(xielu_f(to_float(x[i]), a_pos, a_neg));
}

template <typename T>
__global__ void xielu_vec_kernel(const T* __restrict__ x, T* __restrict__ out, size_t nvec, float a_pos, float a_neg) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= nvec) return;
  float v[Vec<T>::N];
  Vec<T>::load(x + i * Vec<T>::N, v);
#pragma unroll
  for (int j = 0; j < Vec<T>::N; ++j) v[j] = xielu_f(v[j], a_pos, a_neg);
  Vec<T>::store(out + i * Vec<T>::N, v);
}

template <typename T>
__global__ void relu_squared_kernel(const T* __restrict__ x, T* __restrict__ out, size_t n) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float z = fmaxf(to_float(x[i]), 0.f);
  out[i] = from_float<T>(z * z);
}

template <typename T>
__global__ void relu_squared_vec_kernel(const T* __restrict__ x, T* __restrict__ out, size_t nvec) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= nvec) return;
  float v[Vec<T>::N];
  Vec<T>::load(x + i * Vec<T>::N, v);
#pragma unroll
  for (int j = 0; j < Vec<T>::N; ++j) {
    v[j] = fmaxf(v[j], 0.f);
    v[j] *= v[j];
  }
  Vec<T>::store(out + i * Vec<T>::N, v);
}

template <typename T>
__global__ void head_gate_mul_kernel(T* __restrict__ x, const T* __restrict__ g, int64_t ld_g, int col, int heads, int vdim) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int n = heads * vdim;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float gate = 1.0f / (1.0f + expf(-to_float(g[t * ld_g + col + i / vdim])));
    x[t * n + i] = from_float<T>(to_float(x[t * n + i]) * gate);
  }
}

// The same with a gate a number (heads of one value), 16 bytes a thread; a block a token. x and g come from earlier kernels: no __restrict__,
// with which the compiler may load them before pdl_wait().
template <typename T>
__global__ void element_gate_mul_kernel(T* x, const T* g, int64_t ld_g, int col, int n) {
  constexpr int V = Vec<T>::N;
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
    float a[V], b[V];
    Vec<T>::load(x + t * n + i, a);
    Vec<T>::load(g + t * ld_g + col + i, b);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] *= sigmoid_f(b[j]);
    Vec<T>::store(x + t * n + i, a);
  }
}

}  // namespace roost

using namespace roost;

extern "C" int roost_xielu(const void* x, void* out, int64_t n, float a_pos, float a_neg, int dtype, roost_stream_t stream) {
  ROOST_REQUIRE(n >= 0 && (n == 0 || (x && out)), "xielu: a pointer is null");
  if (n == 0) return ROOST_OK;
  const int vec = dtype == ROOST_F32 ? 4 : 8;
  if (n % vec == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)out % 16 == 0) {
    const int64_t nvec = n / vec, blocks = (nvec + 255) / 256;
    if (blocks > 2147483647LL) return fail(ROOST_ERR_UNSUPPORTED, "xielu: too many numbers for one launch");
    ROOST_DISPATCH_DTYPE(dtype, T, launch_kernel(xielu_vec_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, (const T*)x, (T*)out,
                                                 (size_t)nvec, a_pos, a_neg));
    return check_launch("xielu");
  }
  const int64_t blocks = (n + 255) / 256;
  if (blocks > 2147483647LL) return fail(ROOST_ERR_UNSUPPORTED, "xielu: too many numbers for one launch");
  ROOST_DISPATCH_DTYPE(dtype, T, launch_kernel(xielu_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, (const T*)x, (T*)out, (size_t)n,
                                               a_pos, a_neg));
  return check_launch("xielu");
}

extern "C" int roost_relu_squared(const void* x, void* out, int64_t n, int dtype, roost_stream_t stream) {
  ROOST_REQUIRE(n >= 0 && (n == 0 || (x && out)), "relu_squared: a pointer is null");
  if (n == 0) return ROOST_OK;
  const int vec = dtype == ROOST_F32 ? 4 : 8;
  const bool whole = n % vec == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)out % 16 == 0;
  const int64_t items = whole ? n / vec : n, blocks = (items + 255) / 256;
  if (blocks > 2147483647LL) return fail(ROOST_ERR_UNSUPPORTED, "relu_squared: too many numbers for one launch");
  ROOST_DISPATCH_DTYPE(dtype, T, launch_kernel(whole ? relu_squared_vec_kernel<T> : relu_squared_kernel<T>, dim3((unsigned)blocks), dim3(256), 0,
                                               (cudaStream_t)stream, (const T*)x, (T*)out, (size_t)items));
  return check_launch("relu_squared");
}

extern "C" int roost_head_gate_mul(void* x, const void* g, int64_t ld_g, int col, int tokens, int heads, int vdim, int dtype, roost_stream_t stream) {
  ROOST_REQUIRE(tokens >= 0 && heads > 0 && vdim > 0 && col >= 0 && ld_g >= col + heads, "head_gate_mul: sizes do not fit");
  ROOST_REQUIRE(x && g, "head_gate_mul: a pointer is null");
  if (tokens == 0) return ROOST_OK;
  const int vec = dtype == ROOST_F32 ? 4 : 8;
  if (vdim == 1 && heads % vec == 0 && col % vec == 0 && ld_g % vec == 0 && ((uintptr_t)x | (uintptr_t)g) % 16 == 0) {
    const int wide = heads / vec >= 256 ? 256 : (heads / vec >= 128 ? 128 : 64);
    ROOST_DISPATCH_DTYPE(dtype, T, launch_kernel(element_gate_mul_kernel<T>, dim3(tokens), dim3(wide), 0, (cudaStream_t)stream, (T*)x, (const T*)g, ld_g, col,
                                                 heads));
    return check_launch("head_gate_mul");
  }
  const int threads = heads * vdim >= 1024 ? 256 : 128;
  ROOST_DISPATCH_DTYPE(dtype, T, launch_kernel(head_gate_mul_kernel<T>, dim3(tokens), dim3(threads), 0, (cudaStream_t)stream, (T*)x, (const T*)g, ld_g, col,
                                               heads, vdim));
  return check_launch("head_gate_mul");
}
