// Linear attention with a constant decay per head (retention), between the float32 projection [q | k | v] and what the
// output projection reads.  Per head, with q and k rotated at the token's position and k scaled:
//
//   S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   out = o / sqrt(mean(o^2) + eps) * gate(z)
//
// Two forms.  Single tokens: one kernel, a block per (token, head), float32 throughout.  Portions of prompts: chunks of
// 64 tokens of one request.  Inside a chunk everything is a product, only the state's walk from chunk to chunk is a chain:
//
//   chunk_write  U_c = sum_j decay^(n-1-j) k_j v_j^T                                     (a block per chunk and head)
//   chunk_chain  the state before every chunk, in place of its U; the state behind the last goes to its slot
//                S <- decay^n S + U_c, element by element                                (a thread per element)
//   chunk_read   O = ((Q K^T) * decay^(i-j), j <= i) V + decay^(i+1) Q S, norm, gate     (a block per chunk and head)
//
// The products run on the tensor cores (mma.sync.m16n8k16, float32 accumulators).  A read-out that is small is blown up to
// full size by its norm, rounding and all, so every operand (q, k, v, the scores, the state) enters as two bfloat16 parts
// whose sum holds 16 bits of it, in three products (high high, high low, low high).  The state itself is float32.  The
// float32 engine does not use these kernels.
//
// A chunk starts where a tile of the step (at most 128 consecutive tokens of one request) or its second half starts.
// The order of the tiles is the order of the tokens.  States are [seat, head, value_dim, key_dim].  Rotation: a table
// [tokens, rotary_dim] of cosines, then sines, of every token's angles (their factor included), or none.
#include "recurrent.cuh"

namespace distie {

constexpr int kChunk = 64;
constexpr int kReadThreads = 512;    // 16 warps: four groups of 16 rows by four groups of columns
constexpr int kWriteThreads = 256;   // (three blocks an SM)

struct RetentionArgs {
  Sliced qkv;                 // [tokens, heads * (2 * key_dim) + heads * value_dim]
  const float* trig;          // [tokens, rotary_dim] or null
  int rotary_dim, interleaved;
  float key_scale;
  const float* decay;         // [heads]
  float* state;               // [seats, heads, value_dim, key_dim]
  float* chunks;              // [2 * tiles, heads, value_dim, key_dim]
  const int *q_tiles, *token_seq, *seq_seat;
  int tiles, heads, key_dim, value_dim;
};

__device__ __forceinline__ float power_of(float x, int n) {  // x^n, n >= 0
  float out = 1.f;
  for (; n > 0; n >>= 1) {
    if (n & 1) out *= x;
    x *= x;
  }
  return out;
}

// D[16 x 8] += A[16 x 16] B[16 x 8]; with g = lane / 4, c = lane % 4: d = D[g][2c], D[g][2c+1], D[g+8][2c], D[g+8][2c+1].
__device__ __forceinline__ void mma_16bit(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void load_matrices(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void load_matrices_turned(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}

// A matrix in shared memory as two bfloat16 parts, `ld` elements a row; rows start an odd number of 16-byte pieces apart,
// so that the eight rows of an ldmatrix hit different banks.
struct Parts {
  __nv_bfloat16 *high, *low;
  int ld;
  __device__ __forceinline__ void put(int row, int col, float x) const {
    const __nv_bfloat16 h = __float2bfloat16_rn(x);
    high[row * ld + col] = h;
    low[row * ld + col] = __float2bfloat16_rn(x - __bfloat162float(h));
  }
  __device__ __forceinline__ void put2(int row, int col, float x, float y) const {  // col even
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    *reinterpret_cast<__nv_bfloat162*>(high + row * ld + col) = h;
    *reinterpret_cast<__nv_bfloat162*>(low + row * ld + col) =
        __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  }
  __device__ __forceinline__ void put4(int row, int col, float4 x) const {  // col a multiple of 4
    const __nv_bfloat162 h0 = __floats2bfloat162_rn(x.x, x.y), h1 = __floats2bfloat162_rn(x.z, x.w);
    const __nv_bfloat162 l0 = __floats2bfloat162_rn(x.x - __low2float(h0), x.y - __high2float(h0));
    const __nv_bfloat162 l1 = __floats2bfloat162_rn(x.z - __low2float(h1), x.w - __high2float(h1));
    *reinterpret_cast<uint2*>(high + row * ld + col) =
        make_uint2(*reinterpret_cast<const uint32_t*>(&h0), *reinterpret_cast<const uint32_t*>(&h1));
    *reinterpret_cast<uint2*>(low + row * ld + col) =
        make_uint2(*reinterpret_cast<const uint32_t*>(&l0), *reinterpret_cast<const uint32_t*>(&l1));
  }
};
__host__ __device__ constexpr int up16(int n) { return (n + 15) & ~15; }
__host__ __device__ constexpr int parts_ld(int columns) { return up16(columns) + 8; }
__host__ __device__ constexpr size_t parts_bytes(int rows, int columns) { return (size_t)2 * rows * parts_ld(columns) * 2; }
__device__ __forceinline__ Parts parts_at(unsigned char*& at, int rows, int columns) {
  const int ld = parts_ld(columns);
  __nv_bfloat16* p = reinterpret_cast<__nv_bfloat16*>(at);
  at += parts_bytes(rows, columns);
  return Parts{p, p + rows * ld, ld};
}

// The three products of two matrices in parts: `a` 16 rows of the first, `b0`, `b1` eight columns of the second.
__device__ __forceinline__ void mma_parts(float (&d)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1,
                                          uint32_t bl0, uint32_t bl1) {
  mma_16bit(d, ah, bh0, bh1);
  mma_16bit(d, ah, bl0, bl1);
  mma_16bit(d, al, bh0, bh1);
}

// Four neighbours of a projection; WHOLE: it is one matrix, not the slices of a split product.
template <bool WHOLE>
__device__ __forceinline__ float4 four_of(const Sliced& x, size_t t, int col) {
  if (WHOLE) return *reinterpret_cast<const float4*>(x.p + t * x.stride + col);
  return x.at4(t, col);
}

// Rows t0 .. t0 + rows - 1 of one head's q or k (columns from `column`), rotated and times `scale`, into kChunk rows of
// `dst`; rows past the chunk and columns key_dim .. up16(key_dim) - 1 become zeros.
template <bool WHOLE, int kChunkThreads>
__device__ __forceinline__ void load_rotated(const RetentionArgs& a, int t0, int rows, int column, float scale, const Parts& dst) {
  const int half = a.trig ? a.rotary_dim / 2 : 0, rot = 2 * half;
  const int key_dim = a.key_dim, padded = up16(key_dim);
  const bool quads = !a.interleaved && (half & 3) == 0 && (key_dim & 3) == 0 && (a.qkv.stride & 3) == 0 && (column & 3) == 0 &&
                     (a.qkv.split_stride & 3) == 0 && ((uintptr_t)a.qkv.p & 15) == 0 && ((uintptr_t)a.trig & 15) == 0;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  if (quads) {
    const int pairs4 = half / 4, loose4 = (key_dim - rot) / 4, per_row = pairs4 + loose4;
    // A thread keeps its column and takes every r_step-th row.
    const int i = threadIdx.x % per_row, r_step = kChunkThreads / per_row, r_first = threadIdx.x / per_row;
    const int r_end = r_first < r_step ? kChunk : 0;
#pragma unroll 4
    for (int r = r_first; r < r_end; r += r_step) {
      const bool live = r < rows;
      const size_t t = t0 + (live ? r : 0);
      if (i < pairs4) {
        float4 x = zero, y = zero;
        if (live) {
          const float4 u = four_of<WHOLE>(a.qkv, t, column + 4 * i), v = four_of<WHOLE>(a.qkv, t, column + half + 4 * i);
          const float4 cs = *reinterpret_cast<const float4*>(a.trig + t * a.rotary_dim + 4 * i);
          const float4 sn = *reinterpret_cast<const float4*>(a.trig + t * a.rotary_dim + half + 4 * i);
          x = make_float4((u.x * cs.x - v.x * sn.x) * scale, (u.y * cs.y - v.y * sn.y) * scale,
                          (u.z * cs.z - v.z * sn.z) * scale, (u.w * cs.w - v.w * sn.w) * scale);
          y = make_float4((v.x * cs.x + u.x * sn.x) * scale, (v.y * cs.y + u.y * sn.y) * scale,
                          (v.z * cs.z + u.z * sn.z) * scale, (v.w * cs.w + u.w * sn.w) * scale);
        }
        dst.put4(r, 4 * i, x);
        dst.put4(r, half + 4 * i, y);
      } else {
        const int e = rot + 4 * (i - pairs4);
        const float4 x = live ? four_of<WHOLE>(a.qkv, t, column + e) : zero;
        dst.put4(r, e, make_float4(x.x * scale, x.y * scale, x.z * scale, x.w * scale));
      }
    }
  } else {
    const int per_row = key_dim - half;
    for (int idx = threadIdx.x; idx < kChunk * per_row; idx += kChunkThreads) {
      const int r = idx / per_row, i = idx % per_row;
      const bool live = r < rows;
      const size_t t = t0 + (live ? r : 0);
      if (i < half) {
        const int e = a.interleaved ? 2 * i : i, f = a.interleaved ? 2 * i + 1 : i + half;
        float x = 0.f, y = 0.f;
        if (live) {
          const float u = a.qkv.at(t, column + e), v = a.qkv.at(t, column + f);
          const float cs = a.trig[t * a.rotary_dim + i], sn = a.trig[t * a.rotary_dim + half + i];
          x = (u * cs - v * sn) * scale;
          y = (v * cs + u * sn) * scale;
        }
        dst.put(r, e, x);
        dst.put(r, f, y);
      } else {
        dst.put(r, half + i, live ? a.qkv.at(t, column + half + i) * scale : 0.f);
      }
    }
  }
  for (int idx = threadIdx.x; idx < kChunk * (padded - key_dim); idx += kChunkThreads)
    dst.put(idx / (padded - key_dim), key_dim + idx % (padded - key_dim), 0.f);
}

// One head's v of the chunk into kChunk rows of `dst`, row r times weight_s[r] where weights are given; zeros in rows past
// the chunk and in columns value_dim .. up16(value_dim) - 1.
template <bool WHOLE, int kChunkThreads>
__device__ __forceinline__ void load_values(const RetentionArgs& a, int t0, int rows, int column, const float* weight_s, const Parts& dst) {
  const int value_dim = a.value_dim, padded = up16(value_dim);
  const bool quads = (value_dim & 3) == 0 && (a.qkv.stride & 3) == 0 && (column & 3) == 0 && (a.qkv.split_stride & 3) == 0 &&
                     ((uintptr_t)a.qkv.p & 15) == 0;
  if (quads) {
    const int per_row = padded / 4, e = 4 * (threadIdx.x % per_row), r_step = kChunkThreads / per_row;
    const int r_first = threadIdx.x / per_row, r_end = r_first < r_step ? kChunk : 0;
#pragma unroll 4
    for (int r = r_first; r < r_end; r += r_step) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < rows && e < value_dim) x = four_of<WHOLE>(a.qkv, t0 + r, column + e);
      const float w = weight_s ? weight_s[r] : 1.f;
      dst.put4(r, e, make_float4(x.x * w, x.y * w, x.z * w, x.w * w));
    }
  } else {
    for (int idx = threadIdx.x; idx < kChunk * padded; idx += kChunkThreads) {
      const int r = idx / padded, e = idx % padded;
      const float x = r < rows && e < value_dim ? a.qkv.at(t0 + r, column + e) : 0.f;
      dst.put(r, e, weight_s ? x * weight_s[r] : x);
    }
  }
}

// Where chunk `chunk` of the step lies: its first token and its number of tokens (0: the second half of a short tile).
__device__ __forceinline__ int chunk_rows(const int* q_tiles, int chunk, int& t0) {
  const int tile = chunk >> 1, half = chunk & 1;
  t0 = q_tiles[2 * tile] + half * kChunk;
  return min(kChunk, q_tiles[2 * tile + 1] - half * kChunk);
}

// U^T [value_dim, key_dim] of a chunk: rows are value elements (V^T is the first operand), columns key elements.
template <bool WHOLE>
__global__ void __launch_bounds__(kWriteThreads, 3) retention_chunk_write_kernel(RetentionArgs a) {
  extern __shared__ __align__(16) unsigned char chunk_s[];
  __shared__ float weight_s[kChunk];
  int t0;
  const int head = blockIdx.x, rows = chunk_rows(a.q_tiles, blockIdx.y, t0);
  if (rows <= 0) return;
  unsigned char* at = chunk_s;
  const Parts k = parts_at(at, kChunk, a.key_dim), v = parts_at(at, kChunk, a.value_dim);
  const int qk = a.heads * a.key_dim;
  if (threadIdx.x < kChunk) weight_s[threadIdx.x] = threadIdx.x < rows ? power_of(a.decay[head], rows - 1 - threadIdx.x) : 0.f;
  __syncthreads();
  load_rotated<WHOLE, kWriteThreads>(a, t0, rows, qk + head * a.key_dim, a.key_scale, k);
  load_values<WHOLE, kWriteThreads>(a, t0, rows, 2 * qk + head * a.value_dim, weight_s, v);
  __syncthreads();

  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
  const int m_tiles = up16(a.value_dim) / 16, n_tiles = up16(a.key_dim) / 16;
  const int units = m_tiles * ((n_tiles + 1) / 2);  // 16 value elements by 32 key elements each
  float* dst = a.chunks + ((size_t)blockIdx.y * a.heads + head) * a.value_dim * a.key_dim;
  const int steps = (rows + 15) / 16;
  const int v_row = (lane & 7) + (lane >> 4) * 8, v_col = ((lane >> 3) & 1) * 8;  // what a lane names of V^T's 16 x 16 piece
  const int k_row = (lane & 7) + ((lane >> 3) & 1) * 8, k_col = (lane >> 4) * 8;  // and of K's
  for (int unit = warp; unit < units; unit += kWriteThreads / 32) {
    const int m0 = (unit % m_tiles) * 16, n0 = (unit / m_tiles) * 32;
    float acc[4][4] = {};
    for (int s = 0; s < steps; ++s) {
      uint32_t vh[4], vl[4];
      const int v_at = (16 * s + v_row) * v.ld + m0 + v_col;
      load_matrices_turned(vh, v.high + v_at);
      load_matrices_turned(vl, v.low + v_at);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        if (n0 + 16 * j < up16(a.key_dim)) {
          uint32_t kh[4], kl[4];
          const int k_at = (16 * s + k_row) * k.ld + n0 + 16 * j + k_col;
          load_matrices_turned(kh, k.high + k_at);
          load_matrices_turned(kl, k.low + k_at);
          mma_parts(acc[2 * j], vh, vl, kh[0], kh[1], kl[0], kl[1]);
          mma_parts(acc[2 * j + 1], vh, vl, kh[2], kh[3], kl[2], kl[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int row = m0 + g + 8 * h, col = n0 + 8 * j + 2 * c;
        if (row >= a.value_dim || col >= a.key_dim) continue;
        float* to = dst + (size_t)row * a.key_dim + col;
        if ((a.key_dim & 1) == 0) *reinterpret_cast<float2*>(to) = make_float2(acc[j][2 * h], acc[j][2 * h + 1]);
        else {
          to[0] = acc[j][2 * h];
          if (col + 1 < a.key_dim) to[1] = acc[j][2 * h + 1];
        }
      }
    }
  }
}

__device__ __forceinline__ void store_pair(float* p, float x, float y) { *reinterpret_cast<float2*>(p) = make_float2(x, y); }
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float x, float y) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(x, y);
}

// 8 bytes into shared memory, asynchronously; zeros when not live.
__device__ __forceinline__ void copy_8(__nv_bfloat16* dst, const float* src, bool live) {
  const int bytes = live ? 8 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}

// The chain from chunk to chunk of every request: a thread owns W neighbouring elements of one head's state.  What it
// leaves for chunk_read is the state before the chunk in its two bfloat16 parts, in the bytes that held the chunk's U:
// the W high parts, then the W low parts.  A block whose tile is not the first of its request has nothing to do.
constexpr int kChainThreads = 256;
template <int W>
__global__ void __launch_bounds__(kChainThreads) retention_chunk_chain_kernel(RetentionArgs a) {
  const int tile0 = blockIdx.z, head = blockIdx.y;
  const int seq = a.token_seq[a.q_tiles[2 * tile0]];
  if (tile0 > 0 && a.token_seq[a.q_tiles[2 * (tile0 - 1)]] == seq) return;
  const size_t size = (size_t)a.value_dim * a.key_dim;
  const size_t at = ((size_t)blockIdx.x * kChainThreads + threadIdx.x) * W;
  if (at >= size) return;
  struct Piece { float v[W]; };
  auto load = [](const float* p) {
    Piece out;
    if (W == 4) {
      const float4 x = *reinterpret_cast<const float4*>(p);
      out.v[0] = x.x; out.v[W > 1 ? 1 : 0] = x.y; out.v[W > 2 ? 2 : 0] = x.z; out.v[W > 3 ? 3 : 0] = x.w;
    } else {
      out.v[0] = *p;
    }
    return out;
  };
  auto store = [](float* p, const Piece& x) {
    if (W == 4) *reinterpret_cast<float4*>(p) = make_float4(x.v[0], x.v[W > 1 ? 1 : 0], x.v[W > 2 ? 2 : 0], x.v[W > 3 ? 3 : 0]);
    else *p = x.v[0];
  };
  auto store_parts = [](float* p, const Piece& x) {
    if (W == 4) {
      const __nv_bfloat162 h0 = __floats2bfloat162_rn(x.v[0], x.v[W > 1 ? 1 : 0]), h1 = __floats2bfloat162_rn(x.v[W > 2 ? 2 : 0], x.v[W > 3 ? 3 : 0]);
      const __nv_bfloat162 l0 = __floats2bfloat162_rn(x.v[0] - __low2float(h0), x.v[W > 1 ? 1 : 0] - __high2float(h0));
      const __nv_bfloat162 l1 = __floats2bfloat162_rn(x.v[W > 2 ? 2 : 0] - __low2float(h1), x.v[W > 3 ? 3 : 0] - __high2float(h1));
      *reinterpret_cast<uint4*>(p) = make_uint4(*reinterpret_cast<const uint32_t*>(&h0), *reinterpret_cast<const uint32_t*>(&h1),
                                                *reinterpret_cast<const uint32_t*>(&l0), *reinterpret_cast<const uint32_t*>(&l1));
    } else {
      const __nv_bfloat16 h = __float2bfloat16_rn(x.v[0]), l = __float2bfloat16_rn(x.v[0] - __bfloat162float(h));
      *reinterpret_cast<uint32_t*>(p) = (uint32_t)__bfloat16_as_ushort(h) | ((uint32_t)__bfloat16_as_ushort(l) << 16);
    }
  };
  const float decay = a.decay[head], whole = power_of(decay, kChunk);
  float* slot = a.state + ((size_t)a.seq_seat[seq] * a.heads + head) * size + at;
  Piece S = load(slot);
  float* mine = a.chunks + (size_t)head * size + at;
  const size_t stride = (size_t)a.heads * size;
  constexpr int kAhead = 4;  // tiles whose chunks are in flight together
  for (int tile = tile0; tile < a.tiles; tile += kAhead) {
    int rows[kAhead];
    bool more = true;
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      more = more && tile + j < a.tiles && a.token_seq[a.q_tiles[2 * (tile + j)]] == seq;
      rows[j] = more ? a.q_tiles[2 * (tile + j) + 1] : 0;
    }
    Piece u[2 * kAhead];
#pragma unroll
    for (int j = 0; j < 2 * kAhead; ++j)
      if (rows[j >> 1] > (j & 1) * kChunk) u[j] = load(mine + (size_t)(2 * tile + j) * stride);
#pragma unroll
    for (int j = 0; j < 2 * kAhead; ++j) {
      const int n = min(kChunk, rows[j >> 1] - (j & 1) * kChunk);
      if (n > 0) {
        store_parts(mine + (size_t)(2 * tile + j) * stride, S);
        const float factor = n == kChunk ? whole : power_of(decay, n);
#pragma unroll
        for (int e = 0; e < W; ++e) S.v[e] = factor * S.v[e] + u[j].v[e];
      }
    }
    if (!more) break;
  }
  store(slot, S);
}

// O of a chunk from its own tokens and the state before it, normed per head and gated.
template <typename T, bool WHOLE>
__global__ void __launch_bounds__(kReadThreads, 1)
retention_chunk_read_kernel(RetentionArgs a, Sliced gate, int gate_sigmoid, float eps, T* __restrict__ out, int out_stride) {
  extern __shared__ __align__(16) unsigned char chunk_s[];
  __shared__ float power_s[kChunk + 1], square_s[4][kChunk];
  int t0;
  const int head = blockIdx.x, rows = chunk_rows(a.q_tiles, blockIdx.y, t0);
  if (rows <= 0) return;
  const int key_padded = up16(a.key_dim), value_padded = up16(a.value_dim);
  unsigned char* at = chunk_s;
  const Parts q = parts_at(at, kChunk, a.key_dim), k = parts_at(at, kChunk, a.key_dim), v = parts_at(at, kChunk, a.value_dim);
  const Parts S = parts_at(at, value_padded, a.key_dim), p = parts_at(at, kChunk, kChunk);
  const int qk = a.heads * a.key_dim;
  const float* before = a.chunks + ((size_t)blockIdx.y * a.heads + head) * a.value_dim * a.key_dim;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, c = lane & 3;
  const int rg = warp & 3, cq = warp >> 2;   // 16 rows of the chunk; a quarter of the columns
  const int row0 = rg * 16 + g, row1 = row0 + 8;
  const int v0 = cq * 32;                    // the warp's value elements

  if (threadIdx.x <= kChunk) power_s[threadIdx.x] = power_of(a.decay[head], threadIdx.x);
  // The state comes in its two parts already: four elements' high parts, then their low parts, in 16 bytes (or one element's
  // in 4): it is copied while q, k and v are made.
  if ((a.key_dim & 3) == 0) {
    const int per_row = key_padded / 4, e = 4 * (threadIdx.x % per_row), r_step = kReadThreads / per_row;
    const int r_first = threadIdx.x / per_row, r_end = r_first < r_step ? value_padded : 0;
    for (int r = r_first; r < r_end; r += r_step) {
      const bool live = r < a.value_dim && e < a.key_dim;
      const float* src = before + (live ? (size_t)r * a.key_dim + e : 0);
      copy_8(S.high + r * S.ld + e, src, live);
      copy_8(S.low + r * S.ld + e, src + 2, live);
    }
  } else {
    for (int idx = threadIdx.x; idx < value_padded * key_padded; idx += kReadThreads) {
      const int r = idx / key_padded, e = idx % key_padded;
      uint32_t both = 0u;
      if (r < a.value_dim && e < a.key_dim) both = __float_as_uint(before[(size_t)r * a.key_dim + e]);
      S.high[r * S.ld + e] = __ushort_as_bfloat16((unsigned short)(both & 0xffffu));
      S.low[r * S.ld + e] = __ushort_as_bfloat16((unsigned short)(both >> 16));
    }
  }
  cp_async_commit();
  load_rotated<WHOLE, kReadThreads>(a, t0, rows, head * a.key_dim, 1.f, q);
  load_rotated<WHOLE, kReadThreads>(a, t0, rows, qk + head * a.key_dim, a.key_scale, k);
  load_values<WHOLE, kReadThreads>(a, t0, rows, 2 * qk + head * a.value_dim, nullptr, v);
  float z[4][4];  // the gate's inputs of what this thread will store, on their way during the products
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int row = r < 2 ? row0 : row1, col = v0 + 8 * j + 2 * c + (r & 1);
      z[j][r] = 0.f;
      if (row < rows && col < a.value_dim)
        z[j][r] = WHOLE ? gate.p[(size_t)(t0 + row) * gate.stride + head * a.value_dim + col] : gate.at(t0 + row, head * a.value_dim + col);
    }
  cp_async_wait<0>();
  __syncthreads();

  const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;  // what a lane names of a 16 x 16 piece of a
  const int b_row = (lane & 7) + (lane >> 4) * 8, b_col = ((lane >> 3) & 1) * 8;  // first operand, and of a second one by rows
  const int ksteps = key_padded / 16;
  const int q_at = (rg * 16 + a_row) * q.ld + a_col;

  // Scores (16 rows by 16 keys a warp) and what the state before the chunk returns (16 rows by 32 value elements).
  float s[2][4] = {}, o[4][4] = {};
  const bool seen = cq <= rg;  // the warp's keys are not all behind its rows
  for (int step = 0; step < ksteps; ++step) {
    uint32_t qh[4], ql[4], bh[4], bl[4];
    load_matrices(qh, q.high + q_at + 16 * step);
    load_matrices(ql, q.low + q_at + 16 * step);
    if (seen) {
      const int k_at = (cq * 16 + b_row) * k.ld + 16 * step + b_col;
      load_matrices(bh, k.high + k_at);
      load_matrices(bl, k.low + k_at);
      mma_parts(s[0], qh, ql, bh[0], bh[1], bl[0], bl[1]);
      mma_parts(s[1], qh, ql, bh[2], bh[3], bl[2], bl[3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      if (v0 + 16 * j < value_padded) {
        const int s_at = (v0 + 16 * j + b_row) * S.ld + 16 * step + b_col;
        load_matrices(bh, S.high + s_at);
        load_matrices(bl, S.low + s_at);
        mma_parts(o[2 * j], qh, ql, bh[0], bh[1], bl[0], bl[1]);
        mma_parts(o[2 * j + 1], qh, ql, bh[2], bh[3], bl[2], bl[3]);
      }
    }
  }
  // each score times the decay between its two tokens
#pragma unroll
  for (int j = 0; j < 2; ++j) {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int row = h ? row1 : row0, key = cq * 16 + 8 * j + 2 * c;
      p.put2(row, key, key <= row ? s[j][2 * h] * power_s[row - key] : 0.f, key + 1 <= row ? s[j][2 * h + 1] * power_s[row - key - 1] : 0.f);
    }
  }
  const float back0 = power_s[row0 + 1], back1 = power_s[row1 + 1];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    o[j][0] *= back0; o[j][1] *= back0;
    o[j][2] *= back1; o[j][3] *= back1;
  }
  __syncthreads();  // the scores of all columns are in place

  for (int step = 0; step <= rg; ++step) {  // keys up to the warp's last row
    uint32_t ph[4], pw[4];
    const int p_at = (rg * 16 + a_row) * p.ld + 16 * step + a_col;
    load_matrices(ph, p.high + p_at);
    load_matrices(pw, p.low + p_at);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      if (v0 + 16 * j < value_padded) {
        uint32_t bh[4], bl[4];
        const int v_at = (16 * step + a_row) * v.ld + v0 + 16 * j + a_col;
        load_matrices_turned(bh, v.high + v_at);
        load_matrices_turned(bl, v.low + v_at);
        mma_parts(o[2 * j], ph, pw, bh[0], bh[1], bl[0], bl[1]);
        mma_parts(o[2 * j + 1], ph, pw, bh[2], bh[3], bl[2], bl[3]);
      }
    }
  }

  // norm over the head's value elements, gate, store
  float sq0 = 0.f, sq1 = 0.f;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    sq0 += o[j][0] * o[j][0] + o[j][1] * o[j][1];
    sq1 += o[j][2] * o[j][2] + o[j][3] * o[j][3];
  }
#pragma unroll
  for (int offset = 1; offset < 4; offset <<= 1) {
    sq0 += __shfl_xor_sync(0xffffffffu, sq0, offset);
    sq1 += __shfl_xor_sync(0xffffffffu, sq1, offset);
  }
  if (c == 0) {
    square_s[cq][row0] = sq0;
    square_s[cq][row1] = sq1;
  }
  __syncthreads();
  const bool pairs = (a.value_dim & 1) == 0 && (out_stride & 1) == 0 && ((uintptr_t)out & 7) == 0;
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int row = h ? row1 : row0;
    if (row >= rows) continue;
    const float total = (square_s[0][row] + square_s[1][row]) + (square_s[2][row] + square_s[3][row]);
    const float unit = 1.f / sqrtf(total / (float)a.value_dim + eps);
    T* dst = out + (size_t)(t0 + row) * out_stride + head * a.value_dim;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = v0 + 8 * j + 2 * c;
      const float x = o[j][2 * h] * unit * gate_f(gate_sigmoid, z[j][2 * h]);
      const float y = o[j][2 * h + 1] * unit * gate_f(gate_sigmoid, z[j][2 * h + 1]);
      if (pairs && col < a.value_dim) {
        store_pair(dst + col, x, y);
      } else {
        if (col < a.value_dim) dst[col] = from_float<T>(x);
        if (col + 1 < a.value_dim) dst[col + 1] = from_float<T>(y);
      }
    }
  }
}

// Single tokens, a block of eight warps per (head, token): q and k rotated, the state moved on and read, norm and gate.
// A warp owns every eighth row of the head's state (a value element by all key elements); its lanes hold PER key
// elements each, as VEC neighbours (4 or 1) every 32 * VEC.  Rows come kRowsAhead at a time, and the first of them are
// requested before the kernel that makes the projection has finished: nothing between two steps' uses of a request's
// state writes it.  Shared memory: 2 * key_dim + 2 * value_dim floats.
constexpr int kRetentionWarps = 8, kRowsAhead = 4;

template <typename T, int PER, int VEC>
__global__ void __launch_bounds__(kRetentionWarps * 32)
retention_single_kernel(Sliced qkv, Sliced gate, const int* __restrict__ positions, const float* __restrict__ inv_freq, float factor,
                        int rotary_dim, int interleaved, float key_scale, const float* __restrict__ decay, float* state,
                        const int* __restrict__ token_seq, const int* __restrict__ seq_seat, int heads, int key_dim, int value_dim,
                        int gate_sigmoid, float eps, T* out, int out_stride) {
  extern __shared__ __align__(16) float single_s[];
  __shared__ float scratch[32];
  float* q_s = single_s;
  float* k_s = q_s + key_dim;
  float* v_s = k_s + key_dim;
  float* o_s = v_s + value_dim;
  grid_dependency_release();
  const int head = blockIdx.x, t = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int half = inv_freq ? rotary_dim / 2 : 0;
  const float pos = (float)positions[t], g = decay[head];
  float* S = state + ((size_t)seq_seat[token_seq[t]] * heads + head) * value_dim * key_dim;
  auto fetch = [&](int base, float (&rows)[kRowsAhead][PER]) {
#pragma unroll
    for (int r = 0; r < kRowsAhead; ++r) {
      const int j = base + r * kRetentionWarps;
      const float* src = S + (size_t)(j < value_dim ? j : 0) * key_dim;
#pragma unroll
      for (int i = 0; i < PER; i += VEC) {
        const int e = lane * VEC + i * 32;
        const bool live = j < value_dim && e < key_dim;
        if (VEC == 4) {
          const float4 x = live ? load4_cg(src + e) : make_float4(0.f, 0.f, 0.f, 0.f);
          rows[r][i] = x.x; rows[r][i + (VEC > 1 ? 1 : 0)] = x.y; rows[r][i + (VEC > 2 ? 2 : 0)] = x.z; rows[r][i + (VEC > 3 ? 3 : 0)] = x.w;
        } else {
          rows[r][i] = live ? src[e] : 0.f;
        }
      }
    }
  };
  float rows[kRowsAhead][PER];
  fetch(warp, rows);
  // The token's angles: a thread per pair, kept for the head's q and k.
  float cs = 1.f, sn = 0.f;
  const int loose = key_dim - half;  // a thread takes a pair or one of the elements behind them
  if ((int)threadIdx.x < half) {
    sincosf(pos * inv_freq[threadIdx.x], &sn, &cs);
    cs *= factor; sn *= factor;
  }
  grid_dependency_wait();
  const int qk = heads * key_dim;
  const float* row = qkv.p + (size_t)t * qkv.stride;
  const float* z_row = gate.p + (size_t)t * gate.stride + head * value_dim;
  {
    // Everything the thread reads of the projection is requested before any of it is used: a pair (or an element behind
    // the pairs; key_dim <= 256) of q and of k, and its first elements of v and of the gate.
    const int i = threadIdx.x;
    const bool has = i < loose, pair = i < half, value = i < value_dim;
    const int a = pair ? (interleaved ? 2 * i : i) : half + i, b = interleaved ? 2 * i + 1 : i + half;
    const float* q_at = row + head * key_dim;
    const float* k_at = q_at + qk;
    float qa = 0.f, qb = 0.f, ka = 0.f, kb = 0.f, v = 0.f;
    for (int s = 0; s < qkv.splits; s += 4) {
      float d[4][5];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const size_t off = (size_t)(s + u) * qkv.split_stride;
        const bool there = s + u < qkv.splits;
        d[u][0] = there && has ? q_at[off + a] : 0.f;
        d[u][1] = there && pair ? q_at[off + b] : 0.f;
        d[u][2] = there && has ? k_at[off + a] : 0.f;
        d[u][3] = there && pair ? k_at[off + b] : 0.f;
        d[u][4] = there && value ? row[off + 2 * qk + head * value_dim + i] : 0.f;
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) { qa += d[u][0]; qb += d[u][1]; ka += d[u][2]; kb += d[u][3]; v += d[u][4]; }
    }
    if (pair) {
      q_s[a] = qa * cs - qb * sn;
      q_s[b] = qb * cs + qa * sn;
      k_s[a] = (ka * cs - kb * sn) * key_scale;
      k_s[b] = (kb * cs + ka * sn) * key_scale;
    } else if (has) {
      q_s[a] = qa;
      k_s[a] = ka * key_scale;
    }
    if (value) v_s[i] = v;
    for (int e = i + blockDim.x; e < value_dim; e += blockDim.x)
      v_s[e] = sum_slices(row + 2 * qk + head * value_dim + e, qkv.splits, qkv.split_stride);
  }
  const float z_first = (int)threadIdx.x < value_dim ? sum_slices(z_row + threadIdx.x, gate.splits, gate.split_stride) : 0.f;
  __syncthreads();
  float q[PER], k[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = lane * VEC + (i / VEC) * VEC * 32 + i % VEC;
    q[i] = e < key_dim ? q_s[e] : 0.f;
    k[i] = e < key_dim ? k_s[e] : 0.f;
  }
  for (int base = warp; base < value_dim; base += kRowsAhead * kRetentionWarps) {
    float next[kRowsAhead][PER];
    if (base + kRowsAhead * kRetentionWarps < value_dim) fetch(base + kRowsAhead * kRetentionWarps, next);
    float dot[kRowsAhead];
#pragma unroll
    for (int r = 0; r < kRowsAhead; ++r) {
      const int j = base + r * kRetentionWarps;
      const float v = j < value_dim ? v_s[j] : 0.f;
      dot[r] = 0.f;
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        rows[r][i] = g * rows[r][i] + k[i] * v;
        dot[r] += rows[r][i] * q[i];
      }
      if (j < value_dim) {
        float* dst = S + (size_t)j * key_dim;
#pragma unroll
        for (int i = 0; i < PER; i += VEC) {
          const int e = lane * VEC + i * 32;
          if (e < key_dim) {
            if (VEC == 4)
              *reinterpret_cast<float4*>(dst + e) = make_float4(rows[r][i], rows[r][i + (VEC > 1 ? 1 : 0)], rows[r][i + (VEC > 2 ? 2 : 0)],
                                                                rows[r][i + (VEC > 3 ? 3 : 0)]);
            else
              dst[e] = rows[r][i];
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < kRowsAhead; ++r) dot[r] = warp_sum(dot[r]);
    if (lane == 0) {
#pragma unroll
      for (int r = 0; r < kRowsAhead; ++r)
        if (base + r * kRetentionWarps < value_dim) o_s[base + r * kRetentionWarps] = dot[r];
    }
#pragma unroll
    for (int r = 0; r < kRowsAhead; ++r)
#pragma unroll
      for (int i = 0; i < PER; ++i) rows[r][i] = next[r][i];
  }
  __syncthreads();
  float sq = 0.f;
  for (int e = threadIdx.x; e < value_dim; e += blockDim.x) sq += o_s[e] * o_s[e];
  const float unit = 1.f / sqrtf(block_sum(sq, scratch) / (float)value_dim + eps);
  for (int e = threadIdx.x; e < value_dim; e += blockDim.x) {
    const float z = e < (int)blockDim.x ? z_first : sum_slices(z_row + e, gate.splits, gate.split_stride);
    out[(size_t)t * out_stride + head * value_dim + e] = from_float<T>(o_s[e] * unit * gate_f(gate_sigmoid, z));
  }
}

}  // namespace distie

using namespace distie;

// Floats of scratch for the chunks of `tiles` tiles.
extern "C" long long distie_retention_scratch_floats(int tiles, int heads, int key_dim, int value_dim) {
  return 2LL * tiles * heads * key_dim * value_dim;
}

// Portions of prompts: the tokens of `q_tiles` ([tiles, 2] int32: first token, rows <= 128; the tiles of a request follow
// one another).  qkv and gate: float32 projections or their slices.  trig: [tokens, rotary_dim] or null.  out (bfloat16 or
// float32): rows of the tiles' tokens.  -2: sizes these kernels do not take (key_dim and value_dim up to 128).
extern "C" int distie_retention_chunks(const float* qkv, int qkv_stride, int splits, long long split_stride, const float* gate,
                                       int gate_stride, int gate_splits, long long gate_split_stride, const float* trig,
                                       int rotary_dim, int interleaved, float key_scale, const float* decay, float* state,
                                       float* chunks, const int* q_tiles, int tiles, const int* token_seq, const int* seq_seat,
                                       int heads, int key_dim, int value_dim, int gate_sigmoid, float eps, void* out,
                                       int out_stride, int dtype, cudaStream_t stream) {
  if (tiles <= 0) return 0;
  if (heads < 1 || key_dim < 1 || value_dim < 1 || splits < 1 || gate_splits < 1 || !q_tiles || !chunks || !state ||
      (trig && (rotary_dim < 0 || (rotary_dim & 1) || rotary_dim > key_dim)))
    return DISTIE_ERR_ARG;
  if (key_dim > 128 || value_dim > 128 || tiles > 32767 || heads > 65535) return DISTIE_ERR_UNSUPPORTED;
  if (dtype != DISTIE_BF16 && dtype != DISTIE_F32) return DISTIE_ERR_UNSUPPORTED;
  RetentionArgs a{Sliced{qkv, qkv_stride, splits, split_stride}, rotary_dim > 0 ? trig : nullptr, rotary_dim, interleaved, key_scale,
                  decay, state, chunks, q_tiles, token_seq, seq_seat, tiles, heads, key_dim, value_dim};
  const Sliced gates{gate, gate_stride, gate_splits, gate_split_stride};
  const dim3 grid(heads, 2 * tiles);
  const size_t write_shared = parts_bytes(kChunk, key_dim) + parts_bytes(kChunk, value_dim);
  const size_t read_shared = 2 * parts_bytes(kChunk, key_dim) + parts_bytes(kChunk, value_dim) +
                             parts_bytes(up16(value_dim), key_dim) + parts_bytes(kChunk, kChunk);
  auto launch = [&](auto kernel, int threads, size_t shared, auto... args) -> int {
    cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
    if (err != cudaSuccess) return (int)err;
    kernel<<<grid, threads, shared, stream>>>(args...);
    return (int)cudaGetLastError();
  };
  const bool whole = splits == 1 && gate_splits == 1;
  int status = whole ? launch(retention_chunk_write_kernel<true>, kWriteThreads, write_shared, a)
                     : launch(retention_chunk_write_kernel<false>, kWriteThreads, write_shared, a);
  if (status != 0) return status;
  const int size = key_dim * value_dim;
  if (key_dim % 4 == 0)  // (groups of four lie in one row: the layout in which chunk_read takes them)
    retention_chunk_chain_kernel<4><<<dim3((size / 4 + kChainThreads - 1) / kChainThreads, heads, tiles), kChainThreads, 0, stream>>>(a);
  else
    retention_chunk_chain_kernel<1><<<dim3((size + kChainThreads - 1) / kChainThreads, heads, tiles), kChainThreads, 0, stream>>>(a);
  DISTIE_LAUNCH_CHECK();
#define DISTIE_CHUNK_READ(T, WHOLEV) \
  launch(retention_chunk_read_kernel<T, WHOLEV>, kReadThreads, read_shared, a, gates, gate_sigmoid, eps, (T*)out, out_stride)
  if (dtype == DISTIE_BF16) return whole ? DISTIE_CHUNK_READ(__nv_bfloat16, true) : DISTIE_CHUNK_READ(__nv_bfloat16, false);
  return whole ? DISTIE_CHUNK_READ(float, true) : DISTIE_CHUNK_READ(float, false);
#undef DISTIE_CHUNK_READ
}

// The first `count` tokens of the step, each the single token of its request.  -2: sizes not taken (key_dim up to 256).
extern "C" int distie_retention_single(const float* qkv, int qkv_stride, int splits, long long split_stride, const float* gate,
                                       int gate_stride, int gate_splits, long long gate_split_stride, const int* positions,
                                       const float* inv_freq, float factor, int rotary_dim, int interleaved, float key_scale,
                                       const float* decay, float* state, const int* token_seq, const int* seq_seat, int count,
                                       int heads, int key_dim, int value_dim, int gate_sigmoid, float eps, void* out,
                                       int out_stride, int dtype, cudaStream_t stream) {
  if (count <= 0) return 0;
  if (heads < 1 || key_dim < 1 || value_dim < 1 || splits < 1 || gate_splits < 1 || rotary_dim < 0 || (rotary_dim & 1) ||
      rotary_dim > key_dim || (rotary_dim > 0 && !inv_freq))
    return DISTIE_ERR_ARG;
  const size_t shared = 2 * ((size_t)key_dim + value_dim) * sizeof(float);
  if (key_dim > 256 || shared > 48 * 1024 || count > 65535) return DISTIE_ERR_UNSUPPORTED;
  const Sliced rows{qkv, qkv_stride, splits, split_stride}, gates{gate, gate_stride, gate_splits, gate_split_stride};
  const bool vec = key_dim % 4 == 0 && ((uintptr_t)state & 15) == 0;
  cudaError_t err;
#define DISTIE_RETENTION(T, PERV, VECV)                                                                                      \
  err = launch_dependent(retention_single_kernel<T, PERV, VECV>, dim3(heads, count), dim3(kRetentionWarps * 32), shared, stream, \
                         rows, gates, positions, rotary_dim > 0 ? inv_freq : nullptr, factor, rotary_dim, interleaved,      \
                         key_scale, decay, state, token_seq, seq_seat, heads, key_dim, value_dim, gate_sigmoid, eps, (T*)out, \
                         out_stride)
#define DISTIE_RETENTION_SIZES(T)                             \
  do {                                                        \
    if (vec && key_dim <= 128) DISTIE_RETENTION(T, 4, 4);     \
    else if (vec) DISTIE_RETENTION(T, 8, 4);                  \
    else if (key_dim <= 64) DISTIE_RETENTION(T, 2, 1);        \
    else DISTIE_RETENTION(T, 8, 1);                           \
  } while (0)
  if (dtype == DISTIE_BF16) DISTIE_RETENTION_SIZES(__nv_bfloat16);
  else if (dtype == DISTIE_F32) DISTIE_RETENTION_SIZES(float);
  else return DISTIE_ERR_UNSUPPORTED;
#undef DISTIE_RETENTION_SIZES
#undef DISTIE_RETENTION
  return err == cudaSuccess ? 0 : (int)err;
}
