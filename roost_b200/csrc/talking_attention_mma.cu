// The attention of talking_attention.cu on the tensor cores (bfloat16, mma.sync m16n8k16), for steps that bring prompt portions.
//
// One block of 16 warps per (row of the step, 16 of its query tokens, range of up to 16 * OH output heads, chunk of key tiles): all heads' products with a
// tile of 32 keys are needed before any head's softmax, so the block walks the visible keys tile by tile in three phases.
//   own:    a warp a head: S_g = Q_g K^T in 32-bit accumulators, left in shared memory [query][head][key] as float32.
//   mix:    a warp a query: score = scale * (talk S), a product of the matrix talk [heads, heads] (exact in bfloat16: the caller sees to
//           it) with the query's 32-bit S [heads, keys], which enters as three bfloat16 operands (24 bits: all of it); then the mask and
//           the online softmax of every output head, maxima and denominators in registers, the weights as two bfloat16 operands, their
//           rounding and what it left over (16 bits of the 32-bit weights), into the place of S.
//   values: a warp an output head (OH of them): O = O * factor + P V in 32-bit accumulators.
// The next tile's keys are fetched by asynchronous copies while mix and values run, its values while own and mix run; where a tile's keys
// lie in the cache is looked up two tiles ahead. Divided by the denominator, the output gate and the factor come last, then the one
// rounding. A tile of queries with many keys has them dealt to several blocks in chunks of tiles_a_chunk tiles (from its first visible
// key's tile on; the launch's last chunk takes what is left): their sums, maxima and denominators are combined in chunk order by a
// second kernel, so that the blocks of a row's last tiles do not run many times as long as those of its first. Keys outside the block's visible range are not read.
// The queries stay in shared memory where they fit beside the rest; with many heads their fragments come from memory (the caches) instead.
#include "common.cuh"

namespace roost {

constexpr int kTmThreads = 512, kTmWarps = 16;
constexpr int kTmQueries = 16;     // query tokens a block
constexpr int kTmKeys = 32;        // keys a tile
constexpr int kTmSRow = 36;        // floats a head's row of S takes (32 keys, conflict-free reads of eight rows four apart)
constexpr int kTmPlaces = 4;       // tiles whose keys' places in the cache are known: this one and the two after it
constexpr int kTmPRow = 20;        // words a head's row of weights takes (32 bfloat16 and padding)

__device__ __forceinline__ void tm_ldmatrix(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void tm_ldmatrix_trans(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void tm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) rounded to two bfloat16 in one register; x and y become what the rounding left over.
__device__ __forceinline__ uint32_t tm_take(float& x, float& y) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  x -= __bfloat162float(h.x);
  y -= __bfloat162float(h.y);
  return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ void tm_copy16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void tm_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N>
__device__ __forceinline__ void tm_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

// Floats a query's S (and then its weights) takes: 12 modulo 32, so that the eight rows a fragment spans fall in different banks.
__host__ __device__ inline int tm_query_stride(int heads) {
  const int n = heads * 2 * kTmPRow;
  return n + (12 - n % 32 + 32) % 32;
}
__host__ __device__ inline size_t tm_smem_bytes(int heads, int kv_heads, int dim, int vdim, int oh, bool q_staged) {
  const size_t halves = (q_staged ? (size_t)heads * kTmQueries * (dim + 8) : 0) + (size_t)kv_heads * kTmKeys * (dim + vdim + 16) +
                        (size_t)16 * oh * ((heads + 15) / 16 * 16 + 8);
  return halves * 2 + ((size_t)kTmQueries * tm_query_stride(heads) + 2 * (size_t)16 * oh * kTmQueries + kTmPlaces * kTmKeys) * 4;
}

// Which (row, tile of 16 tokens) the block `b` takes: rows in order. False beyond the step's.
__device__ __forceinline__ bool tm_tile_of_block(const int32_t* __restrict__ q_indptr, int rows, int b, int& r, int& k) {
  for (r = 0; r < rows; ++r) {
    const int tiles = (q_indptr[r + 1] - q_indptr[r] + kTmQueries - 1) / kTmQueries;
    if (b < tiles) {
      k = b;
      return true;
    }
    b -= tiles;
  }
  return false;
}

template <int VMAX, int OH>
__global__ void __launch_bounds__(kTmThreads, 1) talking_attention_mma_kernel(
    const __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ out, int64_t ld_out, const __nv_bfloat16* __restrict__ k_base,
    const __nv_bfloat16* __restrict__ v_base, int entry, const __nv_bfloat16* __restrict__ gate, int64_t ld_gate, const float* __restrict__ talk,
    const int32_t* __restrict__ positions, const int32_t* __restrict__ q_indptr, const int32_t* __restrict__ kv_indptr,
    const int32_t* __restrict__ kv_indices, int rows, int heads, int kv_heads, int dim, int vdim, int page_size, float scale, int window,
    float out_scale, int q_staged, float* __restrict__ ws, int tiles_a_chunk, int max_chunks) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  const int ldq = dim + 8, ldv = vdim + 8;                                   // padded rows: ldmatrix without bank conflicts
  const int heads16 = (heads + 15) / 16 * 16, ldt = heads16 + 8;
  const int qs_stride = tm_query_stride(heads);
  __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(sm_raw);              // [head][16][dim + 8]
  __nv_bfloat16* Ks = Qs + (q_staged ? (size_t)heads * kTmQueries * ldq : 0);   // [kv head][32][dim + 8]
  __nv_bfloat16* Vs = Ks + (size_t)kv_heads * kTmKeys * ldq;                 // [kv head][32][vdim + 8]
  __nv_bfloat16* Ts = Vs + (size_t)kv_heads * kTmKeys * ldv;                 // [16 * OH output heads][heads, rounded up to 16]
  float* Ss = reinterpret_cast<float*>(Ts + (size_t)16 * OH * ldt);          // [query][qs_stride]: S, then the weights
  float* Fs = Ss + (size_t)kTmQueries * qs_stride;                           // [output head][query]: the factor on O
  float* Ls = Fs + 16 * OH * kTmQueries;                                     // [output head][query]: the denominator
  int32_t* place = reinterpret_cast<int32_t*>(Ls + 16 * OH * kTmQueries);    // [tile % kTmPlaces][key]: the key's entry for key/value head 0, -1: unseen
  pdl_launch_dependents();
  int r, tile;
  // the blocks with the most keys ahead of them (a row's last tiles) start first
  if (!tm_tile_of_block(q_indptr, rows, (int)gridDim.x - 1 - (int)blockIdx.x, r, tile)) return;
  const int t0 = q_indptr[r] + tile * kTmQueries;
  const int n_valid = min(kTmQueries, q_indptr[r + 1] - t0);
  const int p0 = positions[t0];
  if (p0 < 0) return;                                                        // a padding row
  const int p_last = p0 + n_valid - 1;
  const int lo = window > 0 ? max(0, p0 - window + 1) : 0;                   // the first key any of the queries sees
  const int tile0 = lo / kTmKeys, all = p_last / kTmKeys - tile0 + 1;
  const int chunks = min((all + tiles_a_chunk - 1) / tiles_a_chunk, max_chunks);
  const int z = blockIdx.z;
  if (z >= chunks) return;
  const int first = tile0 + z * tiles_a_chunk, last = z == chunks - 1 ? tile0 + all - 1 : first + tiles_a_chunk - 1;
  const int group = heads / kv_heads;
  const int h0 = blockIdx.y * 16 * OH, hn = min(16 * OH, heads - h0);
  const int32_t* pages = kv_indices + kv_indptr[r];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i < 16 * OH * heads16; i += kTmThreads) {
    const int h = i / heads16, g = i % heads16;
    Ts[h * ldt + g] = __float2bfloat16_rn(h < hn && g < heads ? talk[(size_t)(h0 + h) * heads + g] : 0.f);
  }
  auto place_of = [&](int t) {                                                // of the lane's key of tile t
    const int kp = t * kTmKeys + lane;
    return kp <= p_last && kp >= lo ? pages[kp / page_size] * kv_heads * page_size + kp % page_size : -1;
  };
  if (warp < 2) place[((first + warp) % kTmPlaces) * kTmKeys + lane] = place_of(first + warp);
  __syncthreads();
  pdl_wait();
  // a thread's column of 16 bytes and its first of the (key/value head, key) rows, for keys and for values
  const int k_per = dim / 8, v_per = vdim / 8;
  const int k_row = tid / k_per, k_col = tid % k_per * 8, k_step = kTmThreads / k_per;
  const int v_row = tid / v_per, v_col = tid % v_per * 8, v_step = kTmThreads / v_per;
  auto fetch = [&](__nv_bfloat16* dst, const __nv_bfloat16* base, int ld, int row, int col, int step, int t) {
    const int32_t* at = place + (t % kTmPlaces) * kTmKeys;
    if (row < step)
      for (int gk = row; gk < kv_heads * kTmKeys; gk += step) {
        const int where = at[gk % kTmKeys];                                  // unseen: zeros, nothing is read
        const __nv_bfloat16* src = base;
        if (where >= 0) src += ((size_t)where + (gk / kTmKeys) * page_size) * entry + col;
        tm_copy16((uint32_t)__cvta_generic_to_shared(dst + (size_t)gk * ld + col), src, where >= 0);
      }
    tm_commit();
  };
  if (q_staged) {
    const int per = dim / 8;
    for (int i = tid; i < heads * kTmQueries * per; i += kTmThreads) {
      const int c = i % per, h = (i / per) % heads, n = i / (per * heads);
      const bool live = n < n_valid;
      tm_copy16((uint32_t)__cvta_generic_to_shared(Qs + ((size_t)h * kTmQueries + n) * ldq + c * 8),
                q + ((size_t)(t0 + (live ? n : 0)) * heads + h) * dim + c * 8, live);
    }
  }
  fetch(Ks, k_base, ldq, k_row, k_col, k_step, first);                       // one group with the queries
  fetch(Vs, v_base, ldv, v_row, v_col, v_step, first);
  float o[OH][VMAX / 8][4];
#pragma unroll
  for (int a = 0; a < OH; ++a)
#pragma unroll
    for (int n = 0; n < VMAX / 8; ++n) o[a][n][0] = o[a][n][1] = o[a][n][2] = o[a][n][3] = 0.f;
  float m[OH][2], l[OH][2];                                                  // of output heads lane / 4 and lane / 4 + 8 of each 16, for the warp's query
#pragma unroll
  for (int a = 0; a < OH; ++a) {
    m[a][0] = m[a][1] = -INFINITY;
    l[a][0] = l[a][1] = 0.f;
  }
  const int pos_q = warp < n_valid ? p0 + warp : -1;                         // the query the warp mixes for (-1: sees nothing)
  const int lo_q = window > 0 ? max(0, pos_q - window + 1) : 0;
  const float scale_log2 = scale * 1.4426950408889634f;
  const uint32_t qs_a = (uint32_t)__cvta_generic_to_shared(Qs), ks_a = (uint32_t)__cvta_generic_to_shared(Ks);
  const uint32_t vs_a = (uint32_t)__cvta_generic_to_shared(Vs), ts_a = (uint32_t)__cvta_generic_to_shared(Ts);
  // without staging: the lane's two queries' rows in memory (a query beyond the last: the first one's, nobody reads its results)
  const int n_lo = lane >> 2, n_hi = n_lo + 8;
  const __nv_bfloat16* q_lo = q + (size_t)(t0 + (n_lo < n_valid ? n_lo : 0)) * heads * dim + (lane & 3) * 2;
  const __nv_bfloat16* q_hi = q + (size_t)(t0 + (n_hi < n_valid ? n_hi : 0)) * heads * dim + (lane & 3) * 2;
  float* Sq = Ss + (size_t)warp * qs_stride;
  uint32_t* Pq = reinterpret_cast<uint32_t*>(Sq);                            // [output head][kTmPRow] roundings, then as many remainders
  tm_wait<1>();
  __syncthreads();
  for (int t = first; t <= last; ++t) {
    const int k0 = t * kTmKeys;
    const int ahead = warp == 15 ? place_of(t + 2) : 0;
    // ---- own
    for (int h = warp; h < heads; h += kTmWarps) {
      float c[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n) c[n][0] = c[n][1] = c[n][2] = c[n][3] = 0.f;
      const uint32_t qa = qs_a + (uint32_t)((h * kTmQueries + (lane & 15)) * ldq + (lane >> 4) * 8) * 2;
      const uint32_t ka = ks_a + (uint32_t)(((h / group) * kTmKeys + (lane & 7) + (lane >> 4) * 8) * ldq + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
      for (int ks = 0; ks < dim / 16; ++ks) {
        uint32_t a[4], b[4], d[4];
        if (q_staged) {
          tm_ldmatrix(a, qa + ks * 32);
        } else {
          const int at = h * dim + ks * 16;
          a[0] = *reinterpret_cast<const uint32_t*>(q_lo + at);
          a[1] = *reinterpret_cast<const uint32_t*>(q_hi + at);
          a[2] = *reinterpret_cast<const uint32_t*>(q_lo + at + 8);
          a[3] = *reinterpret_cast<const uint32_t*>(q_hi + at + 8);
        }
        tm_ldmatrix(b, ka + ks * 32);
        tm_ldmatrix(d, ka + ks * 32 + 16 * ldq * 2);
        tm_mma(c[0], a, b[0], b[1]);
        tm_mma(c[1], a, b[2], b[3]);
        tm_mma(c[2], a, d[0], d[1]);
        tm_mma(c[3], a, d[2], d[3]);
      }
      float* s_lo = Ss + (size_t)(lane >> 2) * qs_stride + h * kTmSRow + (lane & 3) * 2;
      float* s_hi = s_lo + (size_t)8 * qs_stride;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        *reinterpret_cast<float2*>(s_lo + n * 8) = make_float2(c[n][0], c[n][1]);
        *reinterpret_cast<float2*>(s_hi + n * 8) = make_float2(c[n][2], c[n][3]);
      }
    }
    __syncthreads();                                                         // S is whole; the keys' buffer is free
    if (t < last) fetch(Ks, k_base, ldq, k_row, k_col, k_step, t + 1);
    else tm_commit();
    // ---- mix
    {
      float c[OH][4][4];
#pragma unroll
      for (int a = 0; a < OH; ++a)
#pragma unroll
        for (int n = 0; n < 4; ++n) c[a][n][0] = c[a][n][1] = c[a][n][2] = c[a][n][3] = 0.f;
      for (int ks = 0; ks < heads16 / 16; ++ks) {
        uint32_t a[OH][4];
#pragma unroll
        for (int i = 0; i < OH; ++i)
          tm_ldmatrix(a[i], ts_a + (uint32_t)((i * 16 + (lane & 15)) * ldt + ks * 16 + (lane >> 4) * 8) * 2);
        const int g = ks * 16 + (lane & 3) * 2;                              // the lane's heads: g, g + 1, g + 8, g + 9
        const float* sg = Sq + g * kTmSRow + (lane >> 2);
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          float s0 = g < heads ? sg[n * 8] : 0.f, s1 = g + 1 < heads ? sg[kTmSRow + n * 8] : 0.f;
          float s8 = g + 8 < heads ? sg[8 * kTmSRow + n * 8] : 0.f, s9 = g + 9 < heads ? sg[9 * kTmSRow + n * 8] : 0.f;
#pragma unroll
          for (int term = 0; term < 3; ++term) {
            const uint32_t b0 = tm_take(s0, s1), b1 = tm_take(s8, s9);
#pragma unroll
            for (int i = 0; i < OH; ++i) tm_mma(c[i][n], a[i], b0, b1);
          }
        }
      }
      __syncwarp();                                                          // every lane has read the query's S: its place takes the weights
#pragma unroll
      for (int i = 0; i < OH; ++i) {
        float mx[2] = {-INFINITY, -INFINITY};
        if (k0 + kTmKeys - 1 <= pos_q && k0 >= lo_q) {                       // the query sees the whole tile
#pragma unroll
          for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              c[i][n][e] *= scale_log2;
              mx[e >> 1] = fmaxf(mx[e >> 1], c[i][n][e]);
            }
        } else {
#pragma unroll
          for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int j = k0 + n * 8 + (lane & 3) * 2 + (e & 1);
              const float v = j <= pos_q && j >= lo_q ? c[i][n][e] * scale_log2 : -INFINITY;
              c[i][n][e] = v;
              mx[e >> 1] = fmaxf(mx[e >> 1], v);
            }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          mx[half] = fmaxf(mx[half], __shfl_xor_sync(0xffffffffu, mx[half], 1));
          mx[half] = fmaxf(mx[half], __shfl_xor_sync(0xffffffffu, mx[half], 2));
          const float m_new = fmaxf(m[i][half], mx[half]);
          const float safe = m_new == -INFINITY ? 0.f : m_new;               // no key seen yet: every weight is 0
          const float keep = exp2f(m[i][half] - safe);
          m[i][half] = m_new;
          float sum = 0.f;
          const int hl = i * 16 + (lane >> 2) + half * 8;
          uint32_t* row = Pq + hl * kTmPRow + (lane & 3);
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            float x = exp2f(c[i][n][2 * half] - safe), y = exp2f(c[i][n][2 * half + 1] - safe);
            sum += x + y;
            const uint32_t hi = tm_take(x, y), rest = tm_take(x, y);
            if (hl < hn) {
              row[n * 4] = hi;
              row[hn * kTmPRow + n * 4] = rest;
            }
          }
          sum += __shfl_xor_sync(0xffffffffu, sum, 1);
          sum += __shfl_xor_sync(0xffffffffu, sum, 2);
          l[i][half] = l[i][half] * keep + sum;
          if ((lane & 3) == 0 && hl < hn) Fs[hl * kTmQueries + warp] = keep;
        }
      }
    }
    if (warp == 15) place[((t + 2) % kTmPlaces) * kTmKeys + lane] = ahead;
    tm_wait<1>();                                                            // the tile's values
    __syncthreads();
    // ---- values
#pragma unroll
    for (int i = 0; i < OH; ++i) {
      const int hl = warp + i * kTmWarps;
      if (hl < hn) {
        const float f0 = Fs[hl * kTmQueries + (lane >> 2)], f1 = Fs[hl * kTmQueries + (lane >> 2) + 8];
        if (__any_sync(0xffffffffu, f0 != 1.0f || f1 != 1.0f)) {
#pragma unroll
          for (int n = 0; n < VMAX / 8; ++n) {
            o[i][n][0] *= f0;
            o[i][n][1] *= f0;
            o[i][n][2] *= f1;
            o[i][n][3] *= f1;
          }
        }
        const uint32_t* p_lo = reinterpret_cast<const uint32_t*>(Ss + (size_t)(lane >> 2) * qs_stride) + hl * kTmPRow + (lane & 3);
        const uint32_t* p_hi = p_lo + (size_t)8 * qs_stride;
        const uint32_t va = vs_a + (uint32_t)((((h0 + hl) / group) * kTmKeys + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int kk = 0; kk < kTmKeys / 16; ++kk) {
          const uint32_t a[4] = {p_lo[kk * 8], p_hi[kk * 8], p_lo[kk * 8 + 4], p_hi[kk * 8 + 4]};
          const int rest = hn * kTmPRow + kk * 8;
          const uint32_t b[4] = {p_lo[rest], p_hi[rest], p_lo[rest + 4], p_hi[rest + 4]};
#pragma unroll
          for (int n = 0; n < VMAX / 16; ++n) {
            if (n * 16 < vdim) {
              uint32_t v[4];
              tm_ldmatrix_trans(v, va + (uint32_t)(kk * 16 * ldv + n * 16) * 2);
              tm_mma(o[i][2 * n], a, v[0], v[1]);
              tm_mma(o[i][2 * n + 1], a, v[2], v[3]);
              tm_mma(o[i][2 * n], b, v[0], v[1]);
              tm_mma(o[i][2 * n + 1], b, v[2], v[3]);
            }
          }
        }
      }
    }
    tm_wait<0>();                                                            // the next tile's keys
    __syncthreads();                                                         // the weights and the values' buffer are free
    if (t < last) fetch(Vs, v_base, ldv, v_row, v_col, v_step, t + 1);
    else tm_commit();
  }
#pragma unroll
  for (int i = 0; i < OH; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int hl = i * 16 + (lane >> 2) + half * 8;
      if ((lane & 3) == 0 && hl < hn) {
        Ls[hl * kTmQueries + warp] = l[i][half];
        if (chunks > 1 && warp < n_valid) {
          float* dst = ws + (((size_t)(t0 + warp) * heads + h0 + hl) * max_chunks + z) * (vdim + 2) + vdim;
          dst[0] = m[i][half];
          dst[1] = l[i][half];
        }
      }
    }
  if (chunks > 1) {                                                          // the chunk's sums, for the kernel that combines a tile's chunks
#pragma unroll
    for (int i = 0; i < OH; ++i) {
      const int hl = warp + i * kTmWarps;
      if (hl >= hn) continue;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int n_q = (lane >> 2) + half * 8;
        if (n_q >= n_valid) continue;
        float* dst = ws + (((size_t)(t0 + n_q) * heads + h0 + hl) * max_chunks + z) * (vdim + 2) + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < VMAX / 8; ++n)
          if (n * 8 < vdim) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[i][n][2 * half], o[i][n][2 * half + 1]);
      }
    }
    return;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < OH; ++i) {
    const int hl = warp + i * kTmWarps;
    if (hl >= hn) continue;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int n_q = (lane >> 2) + half * 8;
      if (n_q >= n_valid) continue;
      const size_t t = (size_t)(t0 + n_q);
      const float den = Ls[hl * kTmQueries + n_q];
      const float inv = den > 0.f ? out_scale / den : 0.f;
#pragma unroll
      for (int n = 0; n < VMAX / 8; ++n) {
        if (n * 8 < vdim) {
          const size_t c = (size_t)(h0 + hl) * vdim + n * 8 + (lane & 3) * 2;
          float x = o[i][n][2 * half] * inv, y = o[i][n][2 * half + 1] * inv;
          if (gate != nullptr) {
            const __nv_bfloat162 gv = *reinterpret_cast<const __nv_bfloat162*>(gate + t * ld_gate + c);
            x *= sigmoid_f(__bfloat162float(gv.x));
            y *= sigmoid_f(__bfloat162float(gv.y));
          }
          *reinterpret_cast<__nv_bfloat162*>(out + t * ld_out + c) = __floats2bfloat162_rn(x, y);
        }
      }
    }
  }
}

// A warp a (token, head): where the token's tile of queries had its keys in several chunks, their sums in chunk order, then the division, the
// gate, the factor and the one rounding.
__global__ void talking_mma_merge_kernel(const float* __restrict__ ws, __nv_bfloat16* __restrict__ out, int64_t ld_out,
                                         const __nv_bfloat16* __restrict__ gate, int64_t ld_gate, const int32_t* __restrict__ positions,
                                         const int32_t* __restrict__ token_row, const int32_t* __restrict__ q_indptr, int heads, int vdim, int window,
                                         float out_scale, int tiles_a_chunk, int max_chunks) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  if (positions[t] < 0) return;
  const int r = token_row[t];
  const int t0 = q_indptr[r] + (t - q_indptr[r]) / kTmQueries * kTmQueries;
  const int p0 = positions[t0], p_last = p0 + min(kTmQueries, q_indptr[r + 1] - t0) - 1;
  const int all = p_last / kTmKeys - (window > 0 ? max(0, p0 - window + 1) : 0) / kTmKeys + 1;
  const int chunks = min((all + tiles_a_chunk - 1) / tiles_a_chunk, max_chunks);
  if (chunks <= 1) return;                                                   // the attention kernel wrote the token's output itself
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int h = blockIdx.y * (blockDim.x / 32) + warp; h < heads; h += gridDim.y * (blockDim.x / 32)) {
    const float* src = ws + ((size_t)t * heads + h) * max_chunks * (vdim + 2);
    float M = -INFINITY;
    for (int z = 0; z < chunks; ++z) M = fmaxf(M, src[(size_t)z * (vdim + 2) + vdim]);
    float L = 0.f, a[4] = {0.f, 0.f, 0.f, 0.f};
    for (int z = 0; z < chunks; ++z) {
      const float* part = src + (size_t)z * (vdim + 2);
      const float f = exp2f(part[vdim] - M);                                 // 0 for a chunk none of whose keys the query sees
      L = fmaf(part[vdim + 1], f, L);
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (lane + 32 * k < vdim) a[k] = fmaf(part[lane + 32 * k], f, a[k]);
    }
    const float inv = L > 0.f ? out_scale / L : 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int i = lane + 32 * k;
      if (i < vdim) {
        const size_t c = (size_t)h * vdim + i;
        float y = a[k] * inv;
        if (gate != nullptr) y *= sigmoid_f(__bfloat162float(gate[(size_t)t * ld_gate + c]));
        out[(size_t)t * ld_out + c] = __float2bfloat16_rn(y);
      }
    }
  }
}

}  // namespace roost

using namespace roost;

constexpr size_t kTmMaxSmem = 226 * 1024;

extern "C" int roost_talking_attention_mma_supported(int heads, int kv_heads, int dim, int vdim, int entry) {
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || dim % 16 || vdim % 16 || vdim > 128 || entry % 8) return 0;
  return tm_smem_bytes(heads, kv_heads, dim, vdim, vdim <= 64 && heads > 16 ? 2 : 1, false) <= kTmMaxSmem ? 1 : 0;
}

extern "C" int roost_talking_attention_mma(const void* q, void* out, int64_t ld_out, const void* k_base, const void* v_base, int entry, const void* gate,
                                           int64_t ld_gate, const float* talk, const int32_t* positions, const int32_t* q_indptr,
                                           const int32_t* kv_indptr, const int32_t* kv_indices, int tokens, int rows, int heads, int kv_heads, int dim,
                                           int vdim, int page_size, float scale, int window, float out_scale, const int32_t* token_row, float* ws, int tiles_a_chunk,
                                           int max_chunks, roost_stream_t stream) {
  ROOST_REQUIRE(tokens >= 0 && rows >= 0 && page_size > 0 && window >= 0, "talking_attention_mma: sizes must be positive");
  ROOST_REQUIRE(q && out && k_base && v_base && talk && positions && q_indptr && kv_indptr && kv_indices, "talking_attention_mma: a pointer is null");
  if (!roost_talking_attention_mma_supported(heads, kv_heads, dim, vdim, entry))
    return fail(ROOST_ERR_UNSUPPORTED, "talking_attention_mma: sizes no tensor-core form serves");
  ROOST_REQUIRE(ld_out >= (int64_t)heads * vdim && (gate == nullptr || ld_gate >= (int64_t)heads * vdim), "talking_attention_mma: a row is too narrow");
  ROOST_REQUIRE((uintptr_t)q % 16 == 0 && (uintptr_t)k_base % 16 == 0 && (uintptr_t)v_base % 16 == 0 && (uintptr_t)out % 4 == 0 && ld_out % 2 == 0 &&
                    (gate == nullptr || ((uintptr_t)gate % 4 == 0 && ld_gate % 2 == 0)),
                "talking_attention_mma: a pointer is not aligned");
  ROOST_REQUIRE(tiles_a_chunk >= 1 && max_chunks >= 1 && max_chunks <= 65535 && (max_chunks == 1 || (ws != nullptr && token_row != nullptr)),
                "talking_attention_mma: chunks of keys need a workspace for their sums");
  if (tokens == 0 || rows == 0) return ROOST_OK;
  const int oh = vdim <= 64 && heads > 16 ? 2 : 1;
  const bool q_staged = tm_smem_bytes(heads, kv_heads, dim, vdim, oh, true) <= kTmMaxSmem;
  const size_t smem = tm_smem_bytes(heads, kv_heads, dim, vdim, oh, q_staged);
  dim3 grid((tokens + kTmQueries - 1) / kTmQueries + rows, (heads + 16 * oh - 1) / (16 * oh), max_chunks);
#define ROOST_TM_LAUNCH(VMAX, OH)                                                                                                                 \
  do {                                                                                                                                            \
    auto kernel = talking_attention_mma_kernel<VMAX, OH>;                                                                                         \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                                   \
    launch_kernel(kernel, grid, dim3(kTmThreads), smem, (cudaStream_t)stream, (const __nv_bfloat16*)q, (__nv_bfloat16*)out, ld_out,               \
                  (const __nv_bfloat16*)k_base, (const __nv_bfloat16*)v_base, entry, (const __nv_bfloat16*)gate, ld_gate, talk, positions, q_indptr, \
                  kv_indptr, kv_indices, rows, heads, kv_heads, dim, vdim, page_size, scale, window, out_scale, q_staged ? 1 : 0, ws,       \
                  tiles_a_chunk, max_chunks);                                                                                                     \
  } while (0)
  if (vdim <= 64 && oh == 2) ROOST_TM_LAUNCH(64, 2);
  else if (vdim <= 64) ROOST_TM_LAUNCH(64, 1);
  else ROOST_TM_LAUNCH(128, 1);
#undef ROOST_TM_LAUNCH
  if (max_chunks > 1)
    launch_kernel(talking_mma_merge_kernel, dim3(tokens, (heads + 7) / 8), dim3(256), 0, (cudaStream_t)stream, (const float*)ws, (__nv_bfloat16*)out, ld_out,
                  (const __nv_bfloat16*)gate, ld_gate, positions, token_row, q_indptr, heads, vdim, window, out_scale, tiles_a_chunk, max_chunks);
  return check_launch("talking_attention_mma");
}
