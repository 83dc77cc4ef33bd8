// Grouped-query causal attention whose scores are mixed across the heads before the softmax (talking heads), over a paged cache.
//
//   own[g, j] = q_g . k_(g's key/value head), j;  score[h, j] = scale * sum_g talk[h, g] own[g, j];
//   out[h] = (sum_j softmax_j(score[h, :]) v_(h's key/value head), j) * sigmoid(gate[h, :]) * out_scale.
//
// A head's weights need every head's product with a key, so a block takes all the heads of its queries. Queries come prepared
// ([tokens, heads, dim]); keys and values lie in the cache in two planes of one size or one plane of [key | value] entries. With a window a
// query at position p sees the keys p - window + 1 .. p; no page before the first such key's tile is looked up.
//
// This file's first kernel is the 32-bit form over a cache of either dtype (every size; decode steps; float32): one block per (token,
// range of output heads, split). Per tile of key_tile keys (absolute positions) all key/value heads' keys and values are staged in shared
// memory as stored, by 16-byte asynchronous copies where the sizes allow (VEC); a thread a (head, key) forms own in 32-bit, then a
// thread a (output head, key) the mixed score and, with the key_tile lanes of its head, the running maximum and denominator; then a
// thread some (head, VEC columns) the sums. A token's tiles may be dealt to several blocks in ranges (from the first visible key's tile);
// their partial sums, maxima and denominators are combined in split order by a second kernel.
#include "common.cuh"

namespace roost {

constexpr int kTaThreads = 256;
constexpr int kTaMaxOut = 8192;      // (output heads x value columns) a block keeps in registers: 32 a thread

template <int VEC, typename T>
__device__ __forceinline__ void talking_load(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == Vec<T>::N) {
    Vec<T>::load(p, v);
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = to_float(p[j]);
  }
}

// Shared memory of a tile's keys and values, as stored, rows padded by 16 bytes; a multiple of 16 bytes.
__host__ __device__ inline size_t talking_tiles_bytes(int kv_heads, int dim, int vdim, int key_tile, int elem) {
  return ((size_t)kv_heads * key_tile * (dim + vdim + 2 * (16 / elem)) * elem + 15) / 16 * 16;
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kTaThreads) talking_attention_kernel(
    const T* __restrict__ q, T* __restrict__ out, int64_t ld_out, float* __restrict__ part, const T* __restrict__ k_base, const T* __restrict__ v_base,
    int entry, const T* __restrict__ gate, int64_t ld_gate, const float* __restrict__ talk, const int32_t* __restrict__ positions,
    const int32_t* __restrict__ token_row, const int32_t* __restrict__ kv_indptr, const int32_t* __restrict__ kv_indices, int heads, int kv_heads,
    int dim, int vdim, int page_size, float scale, int window, float out_scale, int key_tile, int head_chunk, int splits, int tiles_per_split) {
  constexpr int kPad = 16 / (int)sizeof(T);
  constexpr int kUnits = 32 / VEC;
  extern __shared__ __align__(16) unsigned char sm_raw[];
  const int KT = key_tile, ldk = dim + kPad, ldv = vdim + kPad;
  const int h0 = blockIdx.y * head_chunk, hn = min(head_chunk, heads - h0);
  T* ks = reinterpret_cast<T*>(sm_raw);                                      // [kv head][KT][dim + pad]
  T* vs = ks + (size_t)kv_heads * KT * ldk;                                  // [kv head][KT][vdim + pad]
  float* qs = reinterpret_cast<float*>(sm_raw + talking_tiles_bytes(kv_heads, dim, vdim, KT, (int)sizeof(T)));    // [head][dim rounded to 4]
  const int dq = (dim + 3) / 4 * 4;
  float* own = qs + (size_t)heads * dq;                                      // [head][KT]
  float* ps = own + (size_t)heads * KT;                                      // [output head][KT]
  float* mix = ps + (size_t)head_chunk * KT;                                 // [output head][head], times the scale
  float* ms = mix + (size_t)head_chunk * heads;                              // running maximum, denominator, last factor an output head
  float* ls = ms + head_chunk;
  float* fs = ls + head_chunk;
  pdl_launch_dependents();
  const int t = blockIdx.x, z = blockIdx.z, tid = threadIdx.x;
  const int pos = positions[t];
  if (pos < 0) return;                                                       // a padding token
  const int group = heads / kv_heads;
  const int32_t* pages = kv_indices + kv_indptr[token_row[t]];
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;
  const int n_tiles = pos / KT + 1;
  const int first = lo / KT + z * tiles_per_split;
  const int last = z == splits - 1 ? n_tiles : min(n_tiles, first + tiles_per_split);      // the last split takes what is left
  for (int i = tid; i < hn * heads; i += kTaThreads) mix[i] = talk[(size_t)(h0 + i / heads) * heads + i % heads] * scale;
  for (int i = tid; i < hn; i += kTaThreads) {
    ms[i] = -INFINITY;
    ls[i] = 0.f;
  }
  pdl_wait();
  for (int i = tid; i < heads * dim; i += kTaThreads) qs[(i / dim) * dq + i % dim] = to_float(q[(size_t)t * heads * dim + i]);
  float acc[kUnits][VEC];
#pragma unroll
  for (int n = 0; n < kUnits; ++n)
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[n][j] = 0.f;
  const int vunits = (vdim + VEC - 1) / VEC, units = hn * vunits;            // VEC divides vdim
  for (int tile = first; tile < last; ++tile) {
    const int k0 = tile * KT;
    __syncthreads();                                                         // everybody is done with the last tile
    const int kc = dim / VEC, per = kc + vdim / VEC;
    for (int i = tid; i < kv_heads * KT * per; i += kTaThreads) {
      const int c = i % per, key = (i / per) % KT, g = i / (per * KT);
      const int kp = k0 + key;
      const bool seen = kp <= pos && kp >= lo;
      const bool is_k = c < kc;
      const int col = (is_k ? c : c - kc) * VEC;
      T* dst = is_k ? ks + ((size_t)g * KT + key) * ldk + col : vs + ((size_t)g * KT + key) * ldv + col;
      const T* src = is_k ? k_base : v_base;
      if (seen) src += (((size_t)pages[kp / page_size] * kv_heads + g) * page_size + kp % page_size) * entry + col;
      if constexpr (VEC > 1) {
        const int bytes = seen ? 16 : 0;                                     // an unseen key: zeros, nothing is read
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
      } else {
        *dst = seen ? *src : from_float<T>(0.f);
      }
    }
    if constexpr (VEC > 1) asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();
    for (int i = tid; i < heads * KT; i += kTaThreads) {                     // own products
      const int h = i / KT, key = i % KT;
      const T* kr = ks + ((size_t)(h / group) * KT + key) * ldk;
      const float* qh = qs + (size_t)h * dq;
      float s0 = 0.f, s1 = 0.f;
      for (int d = 0; d < dim; d += VEC) {
        float kv[VEC], qv[VEC];
        talking_load<VEC>(kr + d, kv);
        if constexpr (VEC >= 4) {
#pragma unroll
          for (int j = 0; j < VEC; j += 4) {
            const float4 f = *reinterpret_cast<const float4*>(qh + d + j);
            qv[j] = f.x; qv[j + 1] = f.y; qv[j + 2] = f.z; qv[j + 3] = f.w;
          }
        } else {
          qv[0] = qh[d];
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          if (j & 1) s1 = fmaf(qv[j], kv[j], s1);
          else s0 = fmaf(qv[j], kv[j], s0);
        }
      }
      own[i] = s0 + s1;
    }
    __syncthreads();
    for (int i0 = 0; i0 < hn * KT; i0 += kTaThreads) {                       // mixed scores and the running softmax, KT lanes a head
      const int i = i0 + tid;
      const bool live = i < hn * KT;
      const int h = live ? i / KT : 0, key = i % KT, kp = k0 + key;
      float s = -INFINITY;
      if (live && kp <= pos && kp >= lo) {
        s = 0.f;
        const float* mh = mix + (size_t)h * heads;
        for (int g = 0; g < heads; ++g) s = fmaf(mh[g], own[g * KT + key], s);
      }
      float top = s;
      for (int o = KT / 2; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
      const float m_old = live ? ms[h] : -INFINITY;
      const float m_new = fmaxf(m_old, top);
      const float p = s > -INFINITY ? expf(s - m_new) : 0.f;
      float sum = p;
      for (int o = KT / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      __syncwarp();                                                          // the head's lanes have read ms before one of them writes it
      if (live) {
        ps[i] = p;
        if (key == 0) {
          const float keep = m_old > -INFINITY ? expf(m_old - m_new) : 0.f;
          fs[h] = keep;
          ls[h] = ls[h] * keep + sum;
          ms[h] = m_new;
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < kUnits; ++n) {                                       // the weighted values
      const int unit = tid + n * kTaThreads;
      if (unit < units) {
        const int h = unit / vunits, col = (unit % vunits) * VEC;
        const T* vr = vs + (size_t)((h0 + h) / group) * KT * ldv + col;
        const float* ph = ps + (size_t)h * KT;
        const float keep = fs[h];
#pragma unroll
        for (int j = 0; j < VEC; ++j) acc[n][j] *= keep;
        for (int key = 0; key < KT; ++key) {
          float vv[VEC];
          talking_load<VEC>(vr + (size_t)key * ldv, vv);
          const float p = ph[key];
#pragma unroll
          for (int j = 0; j < VEC; ++j) acc[n][j] = fmaf(p, vv[j], acc[n][j]);
        }
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int n = 0; n < kUnits; ++n) {
    const int unit = tid + n * kTaThreads;
    if (unit < units) {
      const int h = unit / vunits, col = (unit % vunits) * VEC;
      if (part != nullptr) {
        float* dst = part + (((size_t)t * heads + h0 + h) * splits + z) * (vdim + 2);
#pragma unroll
        for (int j = 0; j < VEC; ++j) dst[col + j] = acc[n][j];
        if (col == 0) {
          dst[vdim] = ms[h];
          dst[vdim + 1] = ls[h];
        }
      } else {
        const float inv = ls[h] > 0.f ? out_scale / ls[h] : 0.f;
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          const size_t c = (size_t)(h0 + h) * vdim + col + j;
          float y = acc[n][j] * inv;
          if (gate != nullptr) y *= sigmoid_f(to_float(gate[(size_t)t * ld_gate + c]));
          out[(size_t)t * ld_out + c] = from_float<T>(y);
        }
      }
    }
  }
}

// The partials of a token's head, combined in split order; then the gate, the scale and the one rounding.
template <typename T>
__global__ void talking_merge_kernel(const float* __restrict__ part, T* __restrict__ out, int64_t ld_out, const T* __restrict__ gate, int64_t ld_gate,
                                     const int32_t* __restrict__ positions, int heads, int vdim, int splits, float out_scale) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y;
  if (positions[t] < 0) return;
  const float* src = part + ((size_t)t * heads + h) * splits * (vdim + 2);
  const size_t step = vdim + 2;
  float M = -INFINITY;
#pragma unroll 8
  for (int z = 0; z < splits; ++z) M = fmaxf(M, src[z * step + vdim]);
  for (int i = threadIdx.x; i < vdim; i += blockDim.x) {
    float L = 0.f, a = 0.f;
#pragma unroll 8
    for (int z = 0; z < splits; ++z) {
      const float mz = src[z * step + vdim];
      const float f = mz > -INFINITY ? expf(mz - M) : 0.f;
      L = fmaf(src[z * step + vdim + 1], f, L);
      a = fmaf(src[z * step + i], f, a);
    }
    const size_t c = (size_t)h * vdim + i;
    float y = L > 0.f ? a / L * out_scale : 0.f;
    if (gate != nullptr) y *= sigmoid_f(to_float(gate[(size_t)t * ld_gate + c]));
    out[(size_t)t * ld_out + c] = from_float<T>(y);
  }
}

static int talking_head_chunk(int heads, int vdim) { return heads * vdim <= kTaMaxOut ? heads : kTaMaxOut / vdim; }

static size_t talking_smem(int heads, int kv_heads, int dim, int vdim, int key_tile, int elem) {
  const int chunk = talking_head_chunk(heads, vdim);
  const size_t tiles = talking_tiles_bytes(kv_heads, dim, vdim, key_tile, elem);
  const size_t floats = (size_t)heads * ((dim + 3) / 4 * 4) + (size_t)heads * key_tile + (size_t)chunk * key_tile + (size_t)chunk * heads + 3 * (size_t)chunk;
  return tiles + floats * sizeof(float);
}

constexpr size_t kTaMaxSmem = 224 * 1024;

}  // namespace roost

using namespace roost;

extern "C" int roost_talking_attention_key_tile(int heads, int kv_heads, int dim, int vdim, int dtype) {
  if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || vdim > kTaMaxOut) return 0;
  const int elem = dtype == ROOST_F32 ? 4 : 2;
  for (int kt = 32; kt >= 1; kt /= 2)
    if (talking_smem(heads, kv_heads, dim, vdim, kt, elem) <= kTaMaxSmem) return kt;
  return 0;
}

extern "C" int roost_talking_attention(const void* q, void* out, int64_t ld_out, float* part, const void* k_base, const void* v_base, int entry,
                                       const void* gate, int64_t ld_gate, const float* talk, const int32_t* positions, const int32_t* token_row,
                                       const int32_t* kv_indptr, const int32_t* kv_indices, int tokens, int heads, int kv_heads, int dim, int vdim,
                                       int page_size, float scale, int window, float out_scale, int key_tile, int splits, int tiles_per_split, int dtype,
                                       roost_stream_t stream) {
  ROOST_REQUIRE(tokens >= 0 && heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0 && page_size > 0, "talking_attention: sizes must be positive");
  ROOST_REQUIRE(heads % kv_heads == 0, "talking_attention: the query heads are no multiple of the key/value heads");
  ROOST_REQUIRE(q && out && k_base && v_base && talk && positions && token_row && kv_indptr && kv_indices, "talking_attention: a pointer is null");
  ROOST_REQUIRE(window >= 0 && ld_out >= (int64_t)heads * vdim && (gate == nullptr || ld_gate >= (int64_t)heads * vdim),
                "talking_attention: the window is negative or a row is too narrow");
  ROOST_REQUIRE(splits >= 1 && tiles_per_split >= 1 && (splits == 1 || part != nullptr), "talking_attention: splits need a workspace for their partials");
  ROOST_REQUIRE(key_tile >= 1 && key_tile <= 32 && (key_tile & (key_tile - 1)) == 0, "talking_attention: a tile has 1, 2, 4, 8, 16 or 32 keys");
  const int elem = dtype == ROOST_F32 ? 4 : 2;
  if (vdim > kTaMaxOut) return fail(ROOST_ERR_UNSUPPORTED, "talking_attention: values of more than 8192 numbers");
  const size_t smem = talking_smem(heads, kv_heads, dim, vdim, key_tile, elem);
  if (smem > kTaMaxSmem) return fail(ROOST_ERR_UNSUPPORTED, "talking_attention: the heads do not fit in shared memory");
  const int chunk = talking_head_chunk(heads, vdim), chunks = (heads + chunk - 1) / chunk;
  if (splits > 65535 || chunks > 65535) return fail(ROOST_ERR_UNSUPPORTED, "talking_attention: too many heads or splits");
  if (tokens == 0) return ROOST_OK;
  const int vec = 16 / elem;
  const bool whole = dim % vec == 0 && vdim % vec == 0 && entry % vec == 0 && (uintptr_t)k_base % 16 == 0 && (uintptr_t)v_base % 16 == 0;
  cudaStream_t s = (cudaStream_t)stream;
#define ROOST_TA_LAUNCH(VEC)                                                                                                                      \
  do {                                                                                                                                            \
    auto kernel = talking_attention_kernel<T, VEC>;                                                                                               \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                                   \
    launch_kernel(kernel, dim3(tokens, chunks, splits), dim3(kTaThreads), smem, s, (const T*)q, (T*)out, ld_out, splits > 1 ? part : (float*)nullptr, \
                  (const T*)k_base, (const T*)v_base, entry, (const T*)gate, ld_gate, talk, positions, token_row, kv_indptr, kv_indices, heads, kv_heads, \
                  dim, vdim, page_size, scale, window, out_scale, key_tile, chunk, splits, tiles_per_split);                                      \
  } while (0)
  ROOST_DISPATCH_DTYPE(dtype, T, {
    if (whole) ROOST_TA_LAUNCH((16 / (int)sizeof(T)));
    else ROOST_TA_LAUNCH(1);
    if (splits > 1)
      launch_kernel(talking_merge_kernel<T>, dim3(tokens, heads), dim3(vdim >= 128 ? 128 : (vdim >= 64 ? 64 : 32)), 0, s, (const float*)part, (T*)out, ld_out,
                    (const T*)gate, ld_gate, positions, heads, vdim, splits, out_scale);
  });
#undef ROOST_TA_LAUNCH
  return check_launch("talking_attention");
}
