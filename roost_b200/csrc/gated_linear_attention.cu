// Gated linear attention: a matrix state a head whose rows fade by a factor of their own a token, in 32-bit arithmetic.
//
// Per (row, head), for the row's tokens in order, with q, k (dim numbers), v (vdim numbers) and a decay alpha a key channel:
//   S <- diag(alpha) S + k v^T,   o = S^T q.
// The slot holds, head after head, S: dim x vdim. A token's row of the input projection is [q heads | k heads | v heads | ... | a1 | ...]:
// q is multiplied by q_scale; a1 (rank numbers) makes the decays: z = W a1 + bias (heads x dim), alpha = sigmoid(z)^(1 / tau), formed as
// exp(logsigmoid(z) / tau).
//
// prepare: alpha of every token as float32 [tokens, heads * dim]; a thread a channel, whose row of W it reads once for 8 tokens.
//
// scan, heads of up to 128 keys: a block of W warps per (row, head, 32 W columns of S), a warp 32 columns. Lane (cg, dg) of a warp keeps the
// entries of four columns 4 cg .. 4 cg + 3 and of the keys d = 4 i + dg in registers, so that a staged (k, q, alpha), read by all lanes of its
// dg at once, serves four columns; S^T q is the sum over a quad's four lanes. The next 2 W tokens' inputs travel from memory to registers
// while the current ones are multiplied, and are widened to 32-bit on their way into the other half of the stage. Wider heads: one warp
// (a block) per (row, head, 32 columns), S in shared memory, inputs one token ahead. A step of one token a row forms its decays in the scan
// itself (alpha null): no prepare kernel.
//
// Steps of many tokens cut every row into chunks of 64 tokens that run side by side (three launches): a chunk walked from S = 0 ends
// with S'; a state S before the chunk is P S + S' after it, P the products of the chunk's decays a channel. The first walk leaves every
// chunk's own S' and P, one thread an entry then carries the row's state from chunk to chunk leaving every chunk's true starting state
// in the place of S', and a second walk of every chunk from there writes the outputs and, from a row's last chunk, the slot.
//
// What an earlier kernel of the step writes comes through pointers without __restrict__: with it the compiler may load before pdl_wait().
#include "common.cuh"

#include <type_traits>

namespace roost {

constexpr int kGlaChunkTokens = 64;
constexpr int kGlaPrepareTokens = 8;

__device__ __forceinline__ float gla_decay(float z, float inv_tau) {
  const float log_sigmoid = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
  return expf(log_sigmoid * inv_tau);
}

template <typename T>
__global__ void __launch_bounds__(256) gla_prepare_kernel(const T* u, int64_t ld, int a_col, const T* __restrict__ w,
                                                         const float* __restrict__ bias, float* __restrict__ alpha, int tokens, int channels, int rank,
                                                         float inv_tau) {
  extern __shared__ float rows[];      // [kGlaPrepareTokens][rank]
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * kGlaPrepareTokens;
  const int n = min(kGlaPrepareTokens, tokens - t0);
  for (int i = threadIdx.x; i < n * rank; i += blockDim.x) rows[i] = to_float(u[(size_t)(t0 + i / rank) * ld + a_col + i % rank]);
  __syncthreads();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  float z[kGlaPrepareTokens];
  const float b = bias[c];
#pragma unroll
  for (int j = 0; j < kGlaPrepareTokens; ++j) z[j] = 0.f;
  const T* wc = w + (size_t)c * rank;
  for (int r = 0; r < rank; ++r) {
    const float x = to_float(wc[r]);
#pragma unroll
    for (int j = 0; j < kGlaPrepareTokens; ++j)
      if (j < n) z[j] = fmaf(rows[j * rank + r], x, z[j]);
  }
#pragma unroll
  for (int j = 0; j < kGlaPrepareTokens; ++j)
    if (j < n) alpha[(size_t)(t0 + j) * channels + c] = gla_decay(z[j] + b, inv_tau);
}

// Which (row, chunk) the block `b` of a chunked launch takes: rows in order, each with ceil(tokens / 64) chunks.
__device__ __forceinline__ bool gla_chunk_of_block(const int32_t* __restrict__ q_indptr, int rows, int b, int& r, int& k, int& chunks_of_row) {
  for (r = 0; r < rows; ++r) {
    const int n = q_indptr[r + 1] - q_indptr[r];
    chunks_of_row = (n + kGlaChunkTokens - 1) / kGlaChunkTokens;
    if (b < chunks_of_row) {
      k = b;
      return true;
    }
    b -= chunks_of_row;
  }
  return false;
}

// What makes the decays inside the scan (alpha null): the projection's a1 columns, W, the bias.
template <typename T>
struct GlaGate {
  int a_col;
  const T* w;
  const float* bias;
  int rank;
  float inv_tau;
};

// MODE 0: a row's tokens from the slot, which is written back. MODE 1: one chunk from S = 0, leaving S' in ws[chunk] and, from the first
// columns' block, P in ws_keep[chunk]; a row's last chunk is skipped. MODE 2: one chunk from ws[chunk] (the carry kernel put the chunk's true
// starting state there), writing the outputs; a row's last chunk writes the slot.
template <typename T, int DREG, int W, int MODE>
__global__ void __launch_bounds__(32 * W) gla_tile_kernel(const T* u, int64_t ld, float q_scale, const float* alpha, GlaGate<T> gate, float* out, float* state,
                                                         int64_t state_stride, const int32_t* __restrict__ q_indptr, const int32_t* __restrict__ slots,
                                                         int rows, int heads, int dim, int vdim, float* ws, float* ws_keep) {
  constexpr int NT = 32 * W, TT = 2 * W, DG = DREG / 4, NE = TT * DREG / NT;
  __shared__ float4 kqa[2][TT][DREG];
  __shared__ __align__(16) float vs[2][TT][NT];
  __shared__ float products[NT > DREG ? NT : DREG];
  pdl_launch_dependents();
  int r = blockIdx.x, k = 0, chunks_of_row = 1;
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dg = lane & 3, cg = lane >> 2;
  if (MODE != 0 && !gla_chunk_of_block(q_indptr, rows, blockIdx.x, r, k, chunks_of_row)) return;
  if (MODE == 1 && k == chunks_of_row - 1) return;       // nobody starts from the state a row's last chunk ends with
  int start = q_indptr[r], end = q_indptr[r + 1];
  if (MODE != 0) {
    start += k * kGlaChunkTokens;
    end = min(end, start + kGlaChunkTokens);
  }
  const size_t head_state = (size_t)dim * vdim;
  float* slot = state + (size_t)slots[r] * state_stride + (size_t)h * head_state;
  float* wsh = MODE != 0 ? ws + ((size_t)blockIdx.x * heads + h) * head_state : nullptr;
  const float* hs = MODE == 0 ? slot : wsh;
  const int QK = heads * dim;
  const int col_block = blockIdx.z * NT, col0 = col_block + warp * 32 + cg * 4;
  const bool wide = (vdim & 3) == 0 && ((uintptr_t)slot & 15) == 0 && (MODE == 0 || ((uintptr_t)wsh & 15) == 0);      // four columns at a time
  pdl_wait();
  if (end <= start) return;
  float S[DG][4];
#pragma unroll
  for (int i = 0; i < DG; ++i) {
    const int d = 4 * i + dg;
#pragma unroll
    for (int c = 0; c < 4; ++c) S[i][c] = 0.f;
    if (MODE != 1 && d < dim) {
      const float* src = hs + (size_t)d * vdim + col0;
      if (wide && col0 < vdim) {
        const float4 v = *reinterpret_cast<const float4*>(src);
        S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w;
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (col0 + c < vdim) S[i][c] = src[c];
      }
    }
  }
  // the next stage's inputs on their way: entries e = tid + j NT of [TT tokens][DREG keys], and column tid of every token's values
  float nk[NE], nq[NE], na[NE], nv[TT], prod = 1.0f;
  auto fetch = [&](int t0) {
#pragma unroll
    for (int j = 0; j < NE; ++j) {
      const int e = tid + j * NT, t = t0 + e / DREG, d = e % DREG;
      nk[j] = nq[j] = na[j] = 0.f;
      if (t < end && d < dim) {
        const T* row = u + (size_t)t * ld;
        const int c = h * dim + d;
        nq[j] = to_float(row[c]);
        nk[j] = to_float(row[QK + c]);
        if (MODE != 0 || alpha != nullptr) {
          na[j] = alpha[(size_t)t * QK + c];
        } else {
          float z = 0.f;
          for (int i = 0; i < gate.rank; ++i) z = fmaf(to_float(row[gate.a_col + i]), to_float(gate.w[(size_t)c * gate.rank + i]), z);
          na[j] = gla_decay(z + gate.bias[c], gate.inv_tau);
        }
        if (MODE == 1) prod *= na[j];
      }
    }
#pragma unroll
    for (int j = 0; j < TT; ++j) {
      const int t = t0 + j;
      nv[j] = t < end && col_block + tid < vdim ? to_float(u[(size_t)t * ld + 2 * QK + (size_t)h * vdim + col_block + tid]) : 0.f;
    }
  };
  auto store = [&](int buf) {
#pragma unroll
    for (int j = 0; j < NE; ++j) {
      const int e = tid + j * NT;
      kqa[buf][e / DREG][e % DREG] = make_float4(nk[j], nq[j] * q_scale, na[j], 0.f);
    }
#pragma unroll
    for (int j = 0; j < TT; ++j) vs[buf][j][tid] = nv[j];
  };
  fetch(start);
  store(0);
  __syncthreads();
  const bool live = col_block + warp * 32 < vdim;        // the warp has columns
  int buf = 0;
  for (int t0 = start; t0 < end; t0 += TT, buf ^= 1) {
    const bool more = t0 + TT < end;
    if (more) fetch(t0 + TT);
    if (live) {
      const int n = min(TT, end - t0);
      for (int tt = 0; tt < n; ++tt) {
        const float4 v = *reinterpret_cast<const float4*>(&vs[buf][tt][warp * 32 + cg * 4]);
        float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
        for (int i = 0; i < DG; ++i) {
          const float4 f = kqa[buf][tt][4 * i + dg];
          S[i][0] = fmaf(f.z, S[i][0], f.x * v.x);
          S[i][1] = fmaf(f.z, S[i][1], f.x * v.y);
          S[i][2] = fmaf(f.z, S[i][2], f.x * v.z);
          S[i][3] = fmaf(f.z, S[i][3], f.x * v.w);
          if (MODE != 1) {
            o0 = fmaf(S[i][0], f.y, o0);
            o1 = fmaf(S[i][1], f.y, o1);
            o2 = fmaf(S[i][2], f.y, o2);
            o3 = fmaf(S[i][3], f.y, o3);
          }
        }
        if (MODE != 1) {
          // the quad's sums of four columns, one column left in each lane: lane dg ends with column dg
          const bool b0 = dg & 1, b1 = dg & 2;
          const float m0 = (b0 ? o1 : o0) + __shfl_xor_sync(0xffffffffu, b0 ? o0 : o1, 1);
          const float m1 = (b0 ? o3 : o2) + __shfl_xor_sync(0xffffffffu, b0 ? o2 : o3, 1);
          const float sum = (b1 ? m1 : m0) + __shfl_xor_sync(0xffffffffu, b1 ? m0 : m1, 2);
          if (col0 + dg < vdim) out[(size_t)(t0 + tt) * heads * vdim + (size_t)h * vdim + col0 + dg] = sum;
        }
      }
    }
    if (more) store(buf ^ 1);
    __syncthreads();
  }
  if (MODE == 1 && blockIdx.z == 0) {      // thread tid has multiplied the decays of key tid % DREG at some of the tokens
    float* keep = ws_keep + ((size_t)blockIdx.x * heads + h) * dim;
    if (NT >= DREG) {
      products[tid] = prod;
      __syncthreads();
      if (tid < DREG && tid < dim) {
        float p = products[tid];
        for (int i = tid + DREG; i < NT; i += DREG) p *= products[i];
        keep[tid] = p;
      }
    } else {                                // fewer threads than keys: the staged decays are gone, the products come from alpha itself
      for (int d = tid; d < dim; d += NT) {
        float p = 1.0f;
        for (int t = start; t < end; ++t) p *= alpha[(size_t)t * QK + h * dim + d];
        keep[d] = p;
      }
    }
  }
  if (MODE == 2 && k != chunks_of_row - 1) return;
  float* hd = MODE == 1 ? wsh : slot;                     // where the walk's end goes
  if (!live) return;
#pragma unroll
  for (int i = 0; i < DG; ++i) {
    const int d = 4 * i + dg;
    if (d >= dim) continue;
    float* dst = hd + (size_t)d * vdim + col0;
    if (wide && col0 < vdim) {
      *reinterpret_cast<float4*>(dst) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    } else {
#pragma unroll
      for (int c = 0; c < 4; ++c)
        if (col0 + c < vdim) dst[c] = S[i][c];
    }
  }
}

// Heads of more than 128 keys: S in shared memory after the staging area, [dim][32]. The modes are those of gla_tile_kernel.
template <typename T, int MODE>
__global__ void __launch_bounds__(32) gla_scan_kernel(const T* u, int64_t ld, float q_scale, const float* alpha, GlaGate<T> gate,
                                                     float* out, float* state, int64_t state_stride, const int32_t* __restrict__ q_indptr,
                                                     const int32_t* __restrict__ slots, int rows, int heads, int dim, int vdim, float* ws, float* ws_keep) {
  extern __shared__ float4 sm4[];    // two staging slots of dim (k, q, alpha, -); then S
  constexpr int NN = 32;                                 // entries of q, k and alpha a lane loads (dim <= 1024)
  pdl_launch_dependents();
  int r = blockIdx.x, k = 0, chunks_of_row = 1;
  const int h = blockIdx.y, slice = blockIdx.z;
  const int lane = threadIdx.x;
  const int col = slice * 32 + lane;
  const bool live = col < vdim;
  if (MODE != 0 && !gla_chunk_of_block(q_indptr, rows, blockIdx.x, r, k, chunks_of_row)) return;
  if (MODE == 1 && k == chunks_of_row - 1) return;       // nobody starts from the state a row's last chunk ends with
  int start = q_indptr[r], end = q_indptr[r + 1];
  if (MODE != 0) {
    start += k * kGlaChunkTokens;
    end = min(end, start + kGlaChunkTokens);
  }
  const size_t head_state = (size_t)dim * vdim;
  float* slot = state + (size_t)slots[r] * state_stride + (size_t)h * head_state;
  float* wsh = MODE != 0 ? ws + ((size_t)blockIdx.x * heads + h) * head_state : nullptr;
  const float* hs = MODE == 0 ? slot : wsh;               // where the walk starts from (MODE 1 starts empty)
  float* S = reinterpret_cast<float*>(sm4 + 2 * dim) + lane;      // [dim][32]
  const int QK = heads * dim;
  pdl_wait();
  if (end <= start) return;
  for (int d = 0; d < dim; ++d) S[(size_t)d * 32] = (MODE != 1 && live) ? hs[(size_t)d * vdim + col] : 0.f;
  // the next token's inputs, loaded one token ahead
  float nk[NN], nq[NN], na[NN], prod[NN], nv;
#pragma unroll
  for (int i = 0; i < NN; ++i) prod[i] = 1.0f;
  auto load = [&](int t) {
    const T* row = u + (size_t)t * ld;
#pragma unroll
    for (int i = 0; i < NN; ++i) {
      const int d = lane + 32 * i;
      nq[i] = nk[i] = na[i] = 0.f;
      if (d < dim) {
        const int c = h * dim + d;
        nq[i] = to_float(row[c]);
        nk[i] = to_float(row[QK + c]);
        if (MODE != 0 || alpha != nullptr) {
          na[i] = alpha[(size_t)t * QK + c];
        } else {
          float z = 0.f;
          for (int j = 0; j < gate.rank; ++j) z = fmaf(to_float(row[gate.a_col + j]), to_float(gate.w[(size_t)c * gate.rank + j]), z);
          na[i] = gla_decay(z + gate.bias[c], gate.inv_tau);
        }
      }
    }
    nv = live ? to_float(row[2 * QK + (size_t)h * vdim + col]) : 0.f;
  };
  load(start);
  for (int t = start; t < end; ++t) {
    float4* stage = sm4 + (size_t)(t & 1) * dim;
#pragma unroll
    for (int i = 0; i < NN; ++i) {
      const int d = lane + 32 * i;
      if (d < dim) stage[d] = make_float4(nk[i], nq[i] * q_scale, na[i], 0.f);
      if (MODE == 1) prod[i] *= na[i];
    }
    const float val = nv;
    if (t + 1 < end) load(t + 1);
    __syncwarp();
    float num = 0.f;
    for (int d = 0; d < dim; ++d) {
      const float4 f = stage[d];
      const float s = fmaf(f.z, S[(size_t)d * 32], f.x * val);
      S[(size_t)d * 32] = s;
      if (MODE != 1) num = fmaf(s, f.y, num);
    }
    if (MODE != 1 && live) out[(size_t)t * heads * vdim + (size_t)h * vdim + col] = num;
  }
  if (MODE == 1 && slice == 0) {
    float* keep = ws_keep + ((size_t)blockIdx.x * heads + h) * dim;
#pragma unroll
    for (int i = 0; i < NN; ++i) {
      const int d = lane + 32 * i;
      if (d < dim) keep[d] = prod[i];
    }
  }
  if (MODE == 2 && k != chunks_of_row - 1) return;
  float* hd = MODE == 1 ? wsh : slot;                     // where the walk's end goes
  if (live)
    for (int d = 0; d < dim; ++d) hd[(size_t)d * vdim + col] = S[(size_t)d * 32];
}

// One thread an entry of S of a (row, head): the row's state through its chunks in order. ws[chunk] holds the chunk's own S' on entry
// (all but a row's last chunk) and the state the chunk starts from on exit; ws_keep[chunk] the decays' products a channel. The slot is
// read, not written.
__global__ void gla_carry_kernel(const float* state, int64_t state_stride, float* ws, const float* ws_keep,
                                 const int32_t* __restrict__ q_indptr, const int32_t* __restrict__ slots, int heads, int dim, int vdim) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y;
  const int idx = blockIdx.z * blockDim.x + threadIdx.x;
  const int entries = dim * vdim;
  if (idx >= entries) return;
  int first = 0;
  for (int rr = 0; rr < r; ++rr) first += (q_indptr[rr + 1] - q_indptr[rr] + kGlaChunkTokens - 1) / kGlaChunkTokens;
  const int chunks = (q_indptr[r + 1] - q_indptr[r] + kGlaChunkTokens - 1) / kGlaChunkTokens;
  if (chunks == 0) return;
  float e = state[(size_t)slots[r] * state_stride + (size_t)h * entries + idx];
  const size_t stride = (size_t)heads * entries, keep_stride = (size_t)heads * dim;
  float* w0 = ws + ((size_t)first * heads + h) * entries;
  const float* k0p = ws_keep + ((size_t)first * heads + h) * dim + idx / vdim;
  constexpr int kBatch = 8;       // the chunks' own entries do not depend on e: a batch of loads in flight, then the chain
  for (int k0 = 0; k0 < chunks; k0 += kBatch) {
    float own[kBatch], through[kBatch];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const bool in = k0 + j < chunks - 1;
      own[j] = in ? w0[(size_t)(k0 + j) * stride + idx] : 0.f;
      through[j] = in ? k0p[(size_t)(k0 + j) * keep_stride] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      if (k0 + j < chunks) {
        w0[(size_t)(k0 + j) * stride + idx] = e;            // what chunk k0 + j starts from
        if (k0 + j < chunks - 1) e = fmaf(through[j], e, own[j]);
      }
    }
  }
}

template <typename T>
static int gla_scan_launch(const T* u, int64_t ld, float q_scale, const float* alpha, GlaGate<T> gate, float* out, float* state, int64_t state_stride,
                           const int32_t* q_indptr, const int32_t* slots, int rows, int tokens, int heads, int dim, int vdim, float* ws, float* ws_keep,
                           cudaStream_t s) {
  const int slices = (vdim + 31) / 32;
  const int chunks = roost_gla_scan_chunks(tokens, rows);
#define ROOST_GLA_THREE(LAUNCH)                                                                                                             \
  do {                                                                                                                                      \
    if (ws == nullptr) {                                                                                                                    \
      LAUNCH(0, rows);                                                                                                                      \
    } else {                                                                                                                                \
      LAUNCH(1, chunks);                                                                                                                    \
      launch_kernel(gla_carry_kernel, dim3(rows, heads, (dim * vdim + 255) / 256), dim3(256), 0, s, (const float*)state, state_stride, ws,  \
                    (const float*)ws_keep, q_indptr, slots, heads, dim, vdim);                                                              \
      LAUNCH(2, chunks);                                                                                                                    \
    }                                                                                                                                       \
  } while (0)
  auto tile = [&](auto dreg, auto warps) {
    constexpr int D = decltype(dreg)::value, W = decltype(warps)::value;
#define ROOST_GLA_TILE(MODE, GX)                                                                                                            \
  launch_kernel(gla_tile_kernel<T, D, W, MODE>, dim3((GX), heads, (slices + W - 1) / W), dim3(32 * W), 0, s, u, ld, q_scale, alpha, gate,   \
                out, state, state_stride, q_indptr, slots, rows, heads, dim, vdim, ws, ws_keep)
    ROOST_GLA_THREE(ROOST_GLA_TILE);
#undef ROOST_GLA_TILE
  };
  auto heads_of = [&](auto dreg) {
    if (slices >= 3) tile(dreg, std::integral_constant<int, 4>());
    else if (slices == 2) tile(dreg, std::integral_constant<int, 2>());
    else tile(dreg, std::integral_constant<int, 1>());
  };
  if (dim <= 32) {
    heads_of(std::integral_constant<int, 32>());
  } else if (dim <= 64) {
    heads_of(std::integral_constant<int, 64>());
  } else if (dim <= 128) {
    heads_of(std::integral_constant<int, 128>());
  } else {
    const size_t smem = (size_t)2 * dim * sizeof(float4) + (size_t)dim * 32 * sizeof(float);
#define ROOST_GLA_WALK(MODE, GX)                                                                                                            \
  do {                                                                                                                                      \
    auto kernel = gla_scan_kernel<T, MODE>;                                                                                                 \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                             \
    launch_kernel(kernel, dim3((GX), heads, slices), dim3(32), smem, s, u, ld, q_scale, alpha, gate, out, state, state_stride, q_indptr,    \
                  slots, rows, heads, dim, vdim, ws, ws_keep);                                                                              \
  } while (0)
    ROOST_GLA_THREE(ROOST_GLA_WALK);
#undef ROOST_GLA_WALK
  }
#undef ROOST_GLA_THREE
  return check_launch("gla_scan");
}

}  // namespace roost

using namespace roost;

extern "C" int roost_gla_scan_chunks(int tokens, int rows) { return (tokens + kGlaChunkTokens - 1) / kGlaChunkTokens + rows; }

extern "C" int roost_gla_prepare(const void* u, int64_t ld, int a_col, const void* w, const float* bias, float* alpha, int tokens, int channels, int rank,
                                 float tau, int dtype, roost_stream_t stream) {
  ROOST_REQUIRE(tokens >= 0 && channels > 0 && rank > 0 && tau > 0.f, "gla_prepare: sizes and tau must be positive");
  ROOST_REQUIRE(u && w && bias && alpha, "gla_prepare: a pointer is null");
  ROOST_REQUIRE(a_col >= 0 && ld >= (int64_t)a_col + rank, "gla_prepare: a row is too narrow");
  if (tokens == 0) return ROOST_OK;
  const size_t smem = (size_t)kGlaPrepareTokens * rank * sizeof(float);
  if (smem > 48 * 1024) return fail(ROOST_ERR_UNSUPPORTED, "gla_prepare: a gate rank beyond 1536");
  const int threads = channels >= 256 ? 256 : 64;
  ROOST_DISPATCH_DTYPE(dtype, T, launch_kernel(gla_prepare_kernel<T>, dim3((tokens + kGlaPrepareTokens - 1) / kGlaPrepareTokens, (channels + threads - 1) / threads),
                                               dim3(threads), smem, (cudaStream_t)stream, (const T*)u, ld, a_col, (const T*)w, bias, alpha, tokens, channels,
                                               rank, 1.0f / tau));
  return check_launch("gla_prepare");
}

extern "C" int roost_gla_scan(const void* u, int64_t ld, float q_scale, const float* alpha, int a_col, const void* w, const float* bias, int rank, float tau,
                              float* out, float* state, int64_t state_stride, const int32_t* q_indptr, const int32_t* slots, int rows, int tokens, int heads,
                              int dim, int vdim, float* ws, float* ws_keep, int dtype, roost_stream_t stream) {
  ROOST_REQUIRE(rows >= 0 && tokens >= 0 && heads > 0 && dim > 0 && vdim > 0, "gla_scan: sizes must be positive");
  ROOST_REQUIRE(u && out && state && q_indptr && slots, "gla_scan: a pointer is null");
  ROOST_REQUIRE(alpha != nullptr || (w && bias && rank > 0 && tau > 0.f && a_col >= 0 && ld >= (int64_t)a_col + rank),
                "gla_scan: without decays the scan needs what makes them");
  ROOST_REQUIRE((ws == nullptr) == (ws_keep == nullptr) && (ws == nullptr || alpha != nullptr), "gla_scan: a chunked scan needs both workspaces and the decays");
  ROOST_REQUIRE(ld >= (int64_t)heads * (2 * dim + vdim) && state_stride >= (int64_t)heads * dim * vdim, "gla_scan: a row or a slot is too narrow");
  if (dim > 1024) return fail(ROOST_ERR_UNSUPPORTED, "gla_scan: heads of more than 1024 keys");
  if (heads > 65535 || (vdim + 31) / 32 > 65535) return fail(ROOST_ERR_UNSUPPORTED, "gla_scan: too many heads or values");
  if (rows == 0 || tokens == 0) return ROOST_OK;
  ROOST_DISPATCH_DTYPE(dtype, T, {
    GlaGate<T> gate = {a_col, (const T*)w, bias, rank, tau > 0.f ? 1.0f / tau : 0.f};
    return (gla_scan_launch<T>((const T*)u, ld, q_scale, alpha, gate, out, state, state_stride, q_indptr, slots, rows, tokens, heads, dim, vdim, ws,
                               ws_keep, (cudaStream_t)stream));
  });
}
