// A gated recurrence a channel whose gates read only the current token (the minimal gated recurrent unit), in 32-bit arithmetic.
//
// Per (row, channel c), for the row's tokens in order, from the projection's row [z | x | g] (`width` numbers each):
//   z = sigmoid(z + z_bias), x = x + x_bias, cand = x + 1/2 where x >= 0 and sigmoid(x) where x < 0,
//   S <- (1 - z) S + z cand, out = S silu(g) out_scale, rounded once.
// 1 - z is formed as sigmoid of the negated argument (no cancellation where z is near one). S is read from and written back to the row's
// state slot. A thread a channel; a token's loads do not depend on the recurrence, so the loop is unrolled and the next tokens' loads are
// in flight while S advances.
//
// Steps of many tokens cut every row into chunks of 16 tokens that run side by side (three launches): a chunk walked from S = 0 ends
// with S' and the product P of its (1 - z); a state S before the chunk is P S + S' after it. The first walk leaves (S', P) of every
// chunk, one thread a (row, channel) carries the row's state through the chunks, and a second walk of every chunk from its true starting
// state writes the outputs and, from a row's last chunk, the slot.
#include "common.cuh"

namespace roost {

constexpr int kMgChunkTokens = 16;

// Which (row, chunk) the block `b` of a chunked launch takes: rows in order, each with ceil(tokens / 16) chunks. False beyond them.
__device__ __forceinline__ bool min_gru_chunk_of_block(const int32_t* __restrict__ q_indptr, int rows, int b, int& r, int& k, int& chunks_of_row) {
  for (r = 0; r < rows; ++r) {
    const int n = q_indptr[r + 1] - q_indptr[r];
    chunks_of_row = (n + kMgChunkTokens - 1) / kMgChunkTokens;
    if (b < chunks_of_row) {
      k = b;
      return true;
    }
    b -= chunks_of_row;
  }
  return false;
}

// MODE 0: a thread walks its row's tokens from the slot's state and writes the state back. MODE 1: a thread walks one chunk from S = 0
// and leaves S' and P; a row's last chunk is skipped. MODE 2: a thread walks one chunk from ws_state[chunk] (the carry kernel put the
// chunk's true starting state there) and writes the outputs; a row's last chunk leaves the row's state in the slot.
template <typename T, int MODE>
__global__ void __launch_bounds__(128) min_gru_scan_kernel(const T* __restrict__ u, int64_t ld, T* __restrict__ out, int64_t ld_out,
                                                          const float* __restrict__ z_bias, const float* __restrict__ x_bias, float out_scale,
                                                          float* state, int64_t state_stride, const int32_t* __restrict__ q_indptr,
                                                          const int32_t* __restrict__ slots, int rows, int width, float* ws_state, float* ws_keep) {
  pdl_launch_dependents();
  int r = blockIdx.x, k = 0, chunks_of_row = 1;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= width) return;
  if (MODE != 0 && !min_gru_chunk_of_block(q_indptr, rows, blockIdx.x, r, k, chunks_of_row)) return;
  if (MODE == 1 && k == chunks_of_row - 1) return;       // nobody starts from the state a row's last chunk ends with
  const float bz = z_bias[c], bx = x_bias[c];
  int start = q_indptr[r], end = q_indptr[r + 1];
  if (MODE != 0) {
    start += k * kMgChunkTokens;
    end = min(end, start + kMgChunkTokens);
  }
  float* sp = state + (size_t)slots[r] * state_stride + c;
  pdl_wait();
  if (end <= start) return;
  float S = MODE == 0 ? *sp : (MODE == 1 ? 0.f : ws_state[(size_t)blockIdx.x * width + c]);
  float P = 1.0f;
#pragma unroll 4
  for (int t = start; t < end; ++t) {
    const T* row = u + (size_t)t * ld + c;
    const float az = to_float(row[0]) + bz, x = to_float(row[width]) + bx;
    const float z = sigmoid_f(az), keep = sigmoid_f(-az);
    const float cand = x >= 0.f ? x + 0.5f : sigmoid_f(x);
    S = fmaf(keep, S, z * cand);
    if (MODE == 1) {
      P *= keep;
    } else {
      out[(size_t)t * ld_out + c] = from_float<T>(S * silu_f(to_float(row[2 * (size_t)width])) * out_scale);
    }
  }
  if (MODE == 1) {
    ws_state[(size_t)blockIdx.x * width + c] = S;
    ws_keep[(size_t)blockIdx.x * width + c] = P;
  } else if (MODE == 0 || k == chunks_of_row - 1) {
    *sp = S;
  }
}

// One thread a (row, channel): the row's state through its chunks in order. ws_state[chunk] holds S' on entry (all but a row's last
// chunk) and the state the chunk starts from on exit. The slot is read, not written.
__global__ void min_gru_carry_kernel(const float* state, int64_t state_stride, float* __restrict__ ws_state, const float* __restrict__ ws_keep,
                                     const int32_t* __restrict__ q_indptr, const int32_t* __restrict__ slots, int width) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= width) return;
  int first = 0;
  for (int rr = 0; rr < r; ++rr) first += (q_indptr[rr + 1] - q_indptr[rr] + kMgChunkTokens - 1) / kMgChunkTokens;
  const int chunks = (q_indptr[r + 1] - q_indptr[r] + kMgChunkTokens - 1) / kMgChunkTokens;
  if (chunks == 0) return;
  float S = state[(size_t)slots[r] * state_stride + c];
  constexpr int kBatch = 16;      // the chunks' own states do not depend on S: a batch of loads in flight, then the chain
  for (int k0 = 0; k0 < chunks; k0 += kBatch) {
    float own[kBatch], keep[kBatch];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const bool has = k0 + j < chunks - 1;
      own[j] = has ? ws_state[(size_t)(first + k0 + j) * width + c] : 0.f;
      keep[j] = has ? ws_keep[(size_t)(first + k0 + j) * width + c] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      if (k0 + j < chunks) {
        ws_state[(size_t)(first + k0 + j) * width + c] = S;                  // what chunk k0 + j starts from
        if (k0 + j < chunks - 1) S = fmaf(keep[j], S, own[j]);
      }
    }
  }
}

}  // namespace roost

using namespace roost;

extern "C" int roost_min_gru_scan_chunks(int tokens, int rows) { return (tokens + kMgChunkTokens - 1) / kMgChunkTokens + rows; }

extern "C" int roost_min_gru_scan(const void* u, int64_t ld, void* out, int64_t ld_out, const float* z_bias, const float* x_bias, float out_scale,
                                  float* state, int64_t state_stride, const int32_t* q_indptr, const int32_t* slots, int rows, int tokens, int width,
                                  float* ws_state, float* ws_keep, int dtype, roost_stream_t stream) {
  ROOST_REQUIRE(rows >= 0 && tokens >= 0 && width > 0, "min_gru_scan: sizes must be positive");
  ROOST_REQUIRE(u && out && z_bias && x_bias && state && q_indptr && slots, "min_gru_scan: a pointer is null");
  ROOST_REQUIRE(ld >= 3 * (int64_t)width && ld_out >= width && state_stride >= width, "min_gru_scan: a row or a slot is too narrow");
  ROOST_REQUIRE((ws_state == nullptr) == (ws_keep == nullptr), "min_gru_scan: the chunked form needs both workspaces");
  if (rows == 0 || tokens == 0) return ROOST_OK;
  const int gy = (width + 127) / 128;
  if (gy > 65535) return fail(ROOST_ERR_UNSUPPORTED, "min_gru_scan: too many channels");
  cudaStream_t s = (cudaStream_t)stream;
  ROOST_DISPATCH_DTYPE(dtype, T, {
    if (ws_state == nullptr) {
      launch_kernel(min_gru_scan_kernel<T, 0>, dim3(rows, gy), dim3(128), 0, s, (const T*)u, ld, (T*)out, ld_out, z_bias, x_bias, out_scale, state,
                    state_stride, q_indptr, slots, rows, width, ws_state, ws_keep);
    } else {
      const int chunks = roost_min_gru_scan_chunks(tokens, rows);
      launch_kernel(min_gru_scan_kernel<T, 1>, dim3(chunks, gy), dim3(128), 0, s, (const T*)u, ld, (T*)out, ld_out, z_bias, x_bias, out_scale, state,
                    state_stride, q_indptr, slots, rows, width, ws_state, ws_keep);
      launch_kernel(min_gru_carry_kernel, dim3(rows, gy), dim3(128), 0, s, (const float*)state, state_stride, ws_state, (const float*)ws_keep, q_indptr,
                    slots, width);
      launch_kernel(min_gru_scan_kernel<T, 2>, dim3(chunks, gy), dim3(128), 0, s, (const T*)u, ld, (T*)out, ld_out, z_bias, x_bias, out_scale, state,
                    state_stride, q_indptr, slots, rows, width, ws_state, ws_keep);
    }
  });
  return check_launch("min_gru_scan");
}
