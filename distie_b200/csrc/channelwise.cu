// Recurrences whose decay varies by channel and token: the selective scan (a diagonal state per channel) and the delta
// rule with a decay and a removal rate per key channel (a matrix state per head).
//
// Everything is float32 up to the selective scan's gated read-out, which feeds the next product and is stored as T.
// State is read and written through a token's seat; nothing reads host-side batch data beyond counts that a step's
// layout fixes, so captured decode steps replay these kernels.
#include "recurrent.cuh"
#include "tcgen05.cuh"

namespace distie {

constexpr float kLog2e = 1.4426950408889634f;

// 2^x on the special-function unit (results below the smallest normal number become zero).
__device__ __forceinline__ float exp2_unit(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// 32-bit arithmetic on pairs: one instruction, each half rounded as the single operation is.
typedef unsigned long long Pair;
__device__ __forceinline__ Pair pack2(float lo, float hi) {
  Pair p;
  asm("mov.b64 %0, {%1, %2};" : "=l"(p) : "f"(lo), "f"(hi));
  return p;
}
__device__ __forceinline__ float2 unpack2(Pair p) {
  float2 v;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(v.x), "=f"(v.y) : "l"(p));
  return v;
}
__device__ __forceinline__ Pair mul2(Pair a, Pair b) {
  Pair p;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(p) : "l"(a), "l"(b));
  return p;
}
__device__ __forceinline__ Pair fma2(Pair a, Pair b, Pair c) {
  Pair p;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(p) : "l"(a), "l"(b), "l"(c));
  return p;
}

// ---------------------------------------------------------------------------
// Selective scan.  Per channel c and state n, with d = softplus(dt[t, c] + dt_bias[c]):
//   S[n, c] <- exp(d rates[n, c]) S[n, c] + d x[t, c] B[t, n]
//   out[t, c] = (sum_n S[n, c] C[t, n] + skip[c] x[t, c]) * silu(gate[t, c])
// State layout [seat, n, c]: neighbouring threads hold neighbouring channels.
//
// A channel belongs to LANES threads of one warp, each with PER of its states in registers (LANES * PER >= states; what
// lies beyond has no input and adds nothing).  Tokens come in tiles of 16: the block makes d and d x for its channels
// and copies B and C into shared memory, walks the tile, and finishes it element by element (skip, gate, store).
//
// A long prompt alone would leave most of the machine idle, since only channels run side by side.  Its portion is then
// cut into the step's tiles of 128 tokens (`tiles`: first token and length, a request's tiles in a row), and three
// launches replace the walk: (1) every tile but a request's last from a state of zeros, leaving its state and the sum
// of its steps; (2) the chain over a request's tiles, S <- exp(rate * sum of steps) S + the tile's state, which turns
// every tile's state into the one it starts from; (3) every tile from there, with output; a request's last tile leaves
// the request's state.
// ---------------------------------------------------------------------------
constexpr int kSelectTile = 16, kSelectThreads = 128;
constexpr int kSelectWalk = 0, kSelectLocal = 1, kSelectFinish = 2;

struct SelectArgs {
  const float* x;
  int x_stride;
  Sliced dt, B, C, gate;
  const float *rates, *skip, *dt_bias;
  float* state;
  int out_stride;
  const int *seq_bounds, *seq_seat, *token_seq, *tiles;
  int channels, states, first_row, num_tiles;
  float* tile_state;  // [tiles, states, channels]
  float* tile_steps;  // [tiles, channels]
};

// Four neighbouring columns of a row as the element loop needs them: one 16-byte load (VEC), or what there is of them.
template <bool VEC>
__device__ __forceinline__ float4 load_quad(const Sliced& m, size_t row, int col, int columns) {
  if (VEC) return m.at4(row, col);
  float v[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) v[i] = col + i < columns ? m.at(row, col + i) : 0.f;
  return make_float4(v[0], v[1], v[2], v[3]);
}

template <typename T, int PER, int LANES, int MODE, bool VEC>
__global__ void __launch_bounds__(kSelectThreads) selective_scan_kernel(SelectArgs a, T* __restrict__ out) {
  constexpr int CH = kSelectThreads / LANES;  // channels of the block
  constexpr int PER_WARP = 32 / LANES;        // channels of a warp
  constexpr int NP = PER * LANES;
  constexpr int QUADS = CH / 4;               // runs of four channels
  constexpr int ITEMS = (kSelectTile * QUADS + kSelectThreads - 1) / kSelectThreads;  // (token, run) pairs of a thread
  constexpr int ROWS = (kSelectTile * NP + kSelectThreads - 1) / kSelectThreads;      // numbers of B (and of C) of a thread
  __shared__ __align__(16) float d_s[kSelectTile][CH];  // the step sizes; a token's read-out takes the place of its step
  __shared__ __align__(16) float dx_s[kSelectTile][CH];
  __shared__ __align__(16) float b_s[kSelectTile][NP];
  __shared__ __align__(16) float c_s[kSelectTile][NP];
  const int tid = threadIdx.x, lane = tid & 31;
  const int local = (tid >> 5) * PER_WARP + lane % PER_WARP, part = lane / PER_WARP;
  const int c0 = blockIdx.x * CH, c = c0 + local;
  const bool valid = c < a.channels;
  int first, end, row;
  bool last = true;
  if (MODE == kSelectWalk) {
    row = a.first_row + blockIdx.y;
    first = a.seq_bounds[row];
    end = a.seq_bounds[row + 1];
    if (end <= first) return;
  } else {
    const int tile = blockIdx.y;
    first = a.tiles[2 * tile];
    end = first + a.tiles[2 * tile + 1];
    row = a.token_seq[first];
    last = tile + 1 == a.num_tiles || a.token_seq[a.tiles[2 * tile + 2]] != row;
    if (MODE == kSelectLocal && last) return;
  }
  const size_t plane = (size_t)a.states * a.channels;
  float* held = MODE == kSelectWalk ? a.state + (size_t)a.seq_seat[row] * plane : a.tile_state + blockIdx.y * plane;
  const Sliced x{a.x, a.x_stride, 1, 0};

  // A tile's inputs are on their way while the tile before it is walked.
  float4 dt_r[ITEMS], x_r[ITEMS], x_now[ITEMS], gate_r[ITEMS];
  float b_r[ROWS], c_r[ROWS];
  auto place = [&](int item, int& tok, int& ch) {  // (token, first channel) of a thread's item
    const int idx = item * kSelectThreads + tid;
    tok = idx / QUADS;
    ch = (idx % QUADS) * 4;
  };
  auto fetch = [&](int t0) {
    const int count = min(kSelectTile, end - t0);
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      int tok, ch;
      place(i, tok, ch);
      if (tok < count && c0 + ch < a.channels) {
        dt_r[i] = load_quad<VEC>(a.dt, t0 + tok, c0 + ch, a.channels);
        x_r[i] = load_quad<VEC>(x, t0 + tok, c0 + ch, a.channels);
      }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int idx = i * kSelectThreads + tid, tok = idx / NP, n = idx % NP;
      const bool live = tok < count && n < a.states;
      b_r[i] = live ? a.B.at(t0 + tok, n) : 0.f;
      if (MODE != kSelectLocal) c_r[i] = live ? a.C.at(t0 + tok, n) : 0.f;
    }
  };
  fetch(first);

  Pair S[PER / 2], rate[PER / 2];
#pragma unroll
  for (int i = 0; i < PER / 2; ++i) {
    float s[2], r[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int n = part * PER + 2 * i + e;
      const bool live = valid && n < a.states;
      s[e] = (live && MODE != kSelectLocal) ? held[(size_t)n * a.channels + c] : 0.f;
      r[e] = live ? a.rates[(size_t)n * a.channels + c] * kLog2e : 0.f;
    }
    S[i] = pack2(s[0], s[1]);
    rate[i] = pack2(r[0], r[1]);
  }
  float steps = 0.f;
  for (int t0 = first; t0 < end; t0 += kSelectTile) {
    const int count = min(kSelectTile, end - t0);
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      int tok, ch;
      place(i, tok, ch);
      if (tok >= kSelectTile) continue;
      float4 d = make_float4(0.f, 0.f, 0.f, 0.f), dx = d;
      if (tok < count && c0 + ch < a.channels) {
        float bias[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) bias[e] = (VEC || c0 + ch + e < a.channels) ? a.dt_bias[c0 + ch + e] : 0.f;
        d = make_float4(softplus_f(dt_r[i].x + bias[0]), softplus_f(dt_r[i].y + bias[1]), softplus_f(dt_r[i].z + bias[2]),
                        softplus_f(dt_r[i].w + bias[3]));
        dx = make_float4(d.x * x_r[i].x, d.y * x_r[i].y, d.z * x_r[i].z, d.w * x_r[i].w);
        x_now[i] = x_r[i];
        if (MODE != kSelectLocal) gate_r[i] = load_quad<VEC>(a.gate, t0 + tok, c0 + ch, a.channels);
      }
      *reinterpret_cast<float4*>(&d_s[tok][ch]) = d;
      *reinterpret_cast<float4*>(&dx_s[tok][ch]) = dx;
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int idx = i * kSelectThreads + tid;
      if (kSelectTile * NP % kSelectThreads != 0 && idx >= kSelectTile * NP) continue;
      (&b_s[0][0])[idx] = b_r[i];
      if (MODE != kSelectLocal) (&c_s[0][0])[idx] = c_r[i];
    }
    if (t0 + kSelectTile < end) fetch(t0 + kSelectTile);
    __syncthreads();
#pragma unroll 4
    for (int tok = 0; tok < count; ++tok) {
      const float d = d_s[tok][local], dx = dx_s[tok][local];
      const Pair d2 = pack2(d, d), dx2 = pack2(dx, dx);
      Pair y2 = 0;
#pragma unroll
      for (int q = 0; q < PER / 4; ++q) {
        const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(&b_s[tok][part * PER + 4 * q]);
        ulonglong2 w = make_ulonglong2(0, 0);
        if (MODE != kSelectLocal) w = *reinterpret_cast<const ulonglong2*>(&c_s[tok][part * PER + 4 * q]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 z = unpack2(mul2(d2, rate[2 * q + e]));
          const Pair keep = pack2(exp2_unit(z.x), exp2_unit(z.y));
          S[2 * q + e] = fma2(keep, S[2 * q + e], mul2(dx2, e ? b.y : b.x));
          if (MODE != kSelectLocal) y2 = fma2(S[2 * q + e], e ? w.y : w.x, y2);
        }
      }
      if (MODE == kSelectLocal) {
        steps += d;
      } else {
        const float2 halves = unpack2(y2);
        float y = halves.x + halves.y;
#pragma unroll
        for (int offset = PER_WARP; offset < 32; offset <<= 1) y += __shfl_xor_sync(0xffffffffu, y, offset);
        if (part == 0) d_s[tok][local] = y;  // (the channel's other threads have read the step: they took part in the sum)
      }
    }
    __syncthreads();
    if (MODE != kSelectLocal) {
#pragma unroll
      for (int i = 0; i < ITEMS; ++i) {  // (a thread finishes the items that it fills with the next tile)
        int tok, ch;
        place(i, tok, ch);
        if (tok >= count || c0 + ch >= a.channels) continue;
        const float4 y = *reinterpret_cast<const float4*>(&d_s[tok][ch]);
        float skip[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) skip[e] = (VEC || c0 + ch + e < a.channels) ? a.skip[c0 + ch + e] : 0.f;
        const float4 o = make_float4((y.x + skip[0] * x_now[i].x) * silu_f(gate_r[i].x), (y.y + skip[1] * x_now[i].y) * silu_f(gate_r[i].y),
                                     (y.z + skip[2] * x_now[i].z) * silu_f(gate_r[i].z), (y.w + skip[3] * x_now[i].w) * silu_f(gate_r[i].w));
        T* dst = out + (size_t)(t0 + tok) * a.out_stride + c0 + ch;
        if (VEC) {
          store4(dst, o);
        } else {
          const float v[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (c0 + ch + e < a.channels) dst[e] = from_float<T>(v[e]);
        }
      }
    }
  }
  if (!valid) return;
  if (MODE == kSelectFinish) {
    if (!last) return;
    held = a.state + (size_t)a.seq_seat[row] * plane;
  }
  if (MODE == kSelectLocal && part == 0) a.tile_steps[(size_t)blockIdx.y * a.channels + c] = steps;
#pragma unroll
  for (int i = 0; i < PER / 2; ++i) {
    const float2 s = unpack2(S[i]);
    const int n = part * PER + 2 * i;
    if (n < a.states) held[(size_t)n * a.channels + c] = s.x;
    if (n + 1 < a.states) held[(size_t)(n + 1) * a.channels + c] = s.y;
  }
}

// The chain over the tiles of each request, a thread per (state, channel).
__global__ void __launch_bounds__(256) selective_chain_kernel(SelectArgs a) {
  const size_t plane = (size_t)a.states * a.channels;
  const size_t at = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (at >= plane) return;
  const int c = (int)(at % a.channels);
  const float rate = a.rates[at] * kLog2e;
  float S = 0.f;
  int row = -1;
  constexpr int AHEAD = 8;  // tiles whose loads are in flight together
  for (int base = 0; base < a.num_tiles; base += AHEAD) {
    float left[AHEAD], steps[AHEAD];  // (of a request's last tile: not made, and not used)
    int mine[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int tile = min(base + i, a.num_tiles - 1);
      mine[i] = a.token_seq[a.tiles[2 * tile]];
      left[i] = a.tile_state[tile * plane + at];
      steps[i] = a.tile_steps[(size_t)tile * a.channels + c];
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (base + i >= a.num_tiles) break;
      if (mine[i] != row) S = a.state[(size_t)a.seq_seat[mine[i]] * plane + at];
      row = mine[i];
      a.tile_state[(base + i) * plane + at] = S;
      S = exp2_unit(rate * steps[i]) * S + left[i];
    }
  }
}

template <typename T, int PER, int LANES, bool VEC>
static cudaError_t launch_select_as(const SelectArgs& a, T* out, int rows, bool tiled, cudaStream_t stream) {
  const unsigned blocks = (unsigned)((a.channels + kSelectThreads / LANES - 1) / (kSelectThreads / LANES));
  if (rows > 0) selective_scan_kernel<T, PER, LANES, kSelectWalk, VEC><<<dim3(blocks, rows), kSelectThreads, 0, stream>>>(a, out);
  if (tiled) {
    const dim3 grid(blocks, a.num_tiles);
    selective_scan_kernel<T, PER, LANES, kSelectLocal, VEC><<<grid, kSelectThreads, 0, stream>>>(a, out);
    const size_t plane = (size_t)a.states * a.channels;
    selective_chain_kernel<<<(unsigned)((plane + 255) / 256), 256, 0, stream>>>(a);
    selective_scan_kernel<T, PER, LANES, kSelectFinish, VEC><<<grid, kSelectThreads, 0, stream>>>(a, out);
  }
  return cudaGetLastError();
}

template <typename T, int PER, int LANES>
static cudaError_t launch_select(const SelectArgs& a, T* out, int rows, bool tiled, cudaStream_t stream) {
  auto quads = [](const Sliced& m) { return ((m.stride | m.split_stride) & 3) == 0 && ((uintptr_t)m.p & 15) == 0; };
  const bool vec = a.channels % 4 == 0 && ((a.x_stride | a.out_stride) & 3) == 0 && (((uintptr_t)a.x | (uintptr_t)out) & 15) == 0 &&
                   quads(a.dt) && quads(a.gate);
  return vec ? launch_select_as<T, PER, LANES, true>(a, out, rows, tiled, stream)
             : launch_select_as<T, PER, LANES, false>(a, out, rows, tiled, stream);
}

// Threads per channel: few where many tokens are walked (fewer loads and sums per token), more in steps of single tokens.
template <typename T>
static cudaError_t dispatch_select(const SelectArgs& a, T* out, int rows, bool tiled, int lanes, cudaStream_t stream) {
  if (a.states <= 16) {
    if (lanes == 1) return launch_select<T, 16, 1>(a, out, rows, tiled, stream);
    if (lanes == 4) return launch_select<T, 4, 4>(a, out, rows, tiled, stream);
    return launch_select<T, 8, 2>(a, out, rows, tiled, stream);
  }
  if (a.states <= 32) {
    if (lanes >= 4) return launch_select<T, 8, 4>(a, out, rows, tiled, stream);
    return launch_select<T, 16, 2>(a, out, rows, tiled, stream);
  }
  if (a.states <= 64) return launch_select<T, 16, 4>(a, out, rows, tiled, stream);
  if (a.states <= 128) return launch_select<T, 16, 8>(a, out, rows, tiled, stream);
  return launch_select<T, 16, 16>(a, out, rows, tiled, stream);
}

// ---------------------------------------------------------------------------
// Delta rule with a decay w and a removal rate a per key channel.  Per head, with the unit key u = k / |k| (1e-6 under
// the root), S [key, value]:
//   S <- diag(w) S - (a * u) (u^T S) + k v^T   (the old S on the right);   o = S^T r
// Element by element, with g = (k^T S) / (|k|^2 + 1e-6) per column:  S_i <- w_i S_i + k_i (v - a_i g), and the read-out
// is taken from the state before the write:  o = sum_i r_i w_i S_i + v (r . k) - g (sum_i r_i a_i k_i), so both sums over
// the state run side by side.
//
// Two kernels.  The first is parallel over tokens and leaves, per token and head, one contiguous piece of memory: the
// numbers 1 / (|k|^2 + 1e-6), r . k, sum r a k, then the rows k, w, a, r * w and v, padded with zeros to the walk's width.
// The second walks the tokens: the columns of S (one per value element) never meet, so COLS of them belong to a group of
// LANES threads that share their key channels (lane l holds channels 4 l + 4 LANES q + e), a block of 64 threads owns
// 64 / LANES groups of one head of one request.  Bulk copies bring tiles of tokens into shared memory a tile ahead of the
// walk (one elected thread; the wait on their mbarrier is bounded: when it runs out the kernel sets the error word to 6
// and returns).
// State layout: [seat, head, value element, key channel].
// ---------------------------------------------------------------------------
constexpr float kDecayFactor = 0.6065306597126334f;  // exp(-1/2)
constexpr int kDeltaNumbers = 4, kDeltaRows = 5;     // of a token and head

struct DeltaArgs {
  Sliced proj, decay;  // proj: [r | k | v | rate]
  const float *decay_bias, *rate_bias;
  float* scratch;
  float* state;
  float* out;
  const int *seq_bounds, *seq_seat;
  int tokens, heads, dim, width;  // width: dim rounded up to what the walk is compiled for
  int* error;
  __device__ __forceinline__ float* piece(size_t t, int head) const {
    return scratch + (t * heads + head) * (kDeltaNumbers + kDeltaRows * width);
  }
};

__global__ void __launch_bounds__(128) channel_delta_prepare_kernel(DeltaArgs a) {
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int n = a.heads * a.dim;
  for (int head = blockIdx.y * 4 + warp; head < a.heads; head += gridDim.y * 4) {
    float* numbers = a.piece(t, head);
    float* rows = numbers + kDeltaNumbers;
    float kk = 0.f, rk = 0.f, rak = 0.f;
    for (int i = a.dim + lane; i < a.width; i += 32)
      for (int which = 0; which < kDeltaRows; ++which) rows[which * a.width + i] = 0.f;
    for (int i = lane; i < a.dim; i += 32) {
      const int col = head * a.dim + i;
      const float r = a.proj.at(t, col), k = a.proj.at(t, n + col), v = a.proj.at(t, 2 * n + col);
      const float rate = sigmoid_f(a.proj.at(t, 3 * n + col) + a.rate_bias[col]);
      const float w = expf(-kDecayFactor * sigmoid_f(a.decay.at(t, col) + a.decay_bias[col]));
      rows[i] = k;
      rows[a.width + i] = w;
      rows[2 * a.width + i] = rate;
      rows[3 * a.width + i] = r * w;
      rows[4 * a.width + i] = v;
      kk += k * k;
      rk += r * k;
      rak += r * rate * k;
    }
    kk = warp_sum(kk);
    rk = warp_sum(rk);
    rak = warp_sum(rak);
    if (lane == 0) *reinterpret_cast<float4*>(numbers) = make_float4(1.f / (kk + 1e-6f), rk, rak, 0.f);
  }
}

// One copy of `bytes` (a multiple of 16, both addresses on 16-byte boundaries) into shared memory, counted on `bar`.
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

// The sums of NV values over groups of LANES neighbouring lanes with few exchanges: every round hands half of the values
// to a neighbour and keeps the other half; when one value a lane is left, the rest of the group is summed by butterflies.
// Afterwards v[0] of a lane is the sum of value `value_of(lane)`.
template <int NV, int LANES>
struct FoldedSum {
  __host__ __device__ static constexpr int bits() { return NV == 2 ? 1 : NV == 4 ? 2 : 3; }
  static __device__ __forceinline__ int value_of(int lane) {
    int value = 0;
    for (int b = 0; b < bits(); ++b) value |= ((lane >> b) & 1) << (bits() - 1 - b);
    return value;
  }
  static __device__ __forceinline__ float run(float (&v)[NV], int sub) {
#pragma unroll
    for (int b = 0; b < bits(); ++b) {
      const int half = NV >> (b + 1);
      const bool upper = (sub >> b) & 1;
#pragma unroll
      for (int i = 0; i < NV / 2; ++i) {
        if (i >= half) break;
        const float give = upper ? v[i] : v[i + half], keep = upper ? v[i + half] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1 << b);
      }
    }
#pragma unroll
    for (int offset = 1 << bits(); offset < LANES; offset <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], offset);
    return v[0];
  }
};

template <int KD, int TILE>
struct DeltaStage {
  float piece[TILE][kDeltaNumbers + kDeltaRows * KD];
};

// VEC: columns of the state start on 16-byte boundaries.
template <int KD, int LANES, int COLS, int TILE, int THREADS, bool VEC>
__global__ void __launch_bounds__(THREADS, 256 / THREADS) channel_delta_kernel(DeltaArgs a) {
  constexpr int PER = KD / LANES, CB = THREADS / LANES * COLS;
  using Fold = FoldedSum<TILE, LANES>;  // of a tile's read-outs of one column
  static_assert(PER >= 4 && PER % 4 == 0 && TILE <= LANES, "a thread holds whole float4s of its columns");
  extern __shared__ __align__(16) unsigned char delta_smem[];
  using Stage = DeltaStage<KD, TILE>;
  Stage* stages = reinterpret_cast<Stage*>(delta_smem);  // two
  __shared__ __align__(8) uint64_t full[2];
  const int row = blockIdx.x, head = blockIdx.y;
  const int tid = threadIdx.x, sub = tid % LANES, group = tid / LANES;
  const int j0 = blockIdx.z * CB + group * COLS;
  const int first = a.seq_bounds[row], end = a.seq_bounds[row + 1];
  if (end <= first) return;
  if (tid == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();

  constexpr uint32_t kBytes = (kDeltaNumbers + kDeltaRows * KD) * sizeof(float);
  auto stage_tile = [&](int tile, int buffer) {  // one thread
    const int count = min(TILE, end - tile);
    mbar_expect_tx(&full[buffer], count * kBytes);
    for (int tok = 0; tok < count; ++tok) bulk_load(stages[buffer].piece[tok], a.piece(tile + tok, head), kBytes, &full[buffer]);
  };
  if (tid == 0) stage_tile(first, 0);
  float* held = a.state + ((size_t)a.seq_seat[row] * a.heads + head) * a.dim * a.dim;
  Pair S[COLS][PER / 2];
#pragma unroll
  for (int col = 0; col < COLS; ++col)
#pragma unroll
    for (int q = 0; q < PER / 4; ++q) {
      const int i = 4 * sub + 4 * LANES * q;
      const bool live = j0 + col < a.dim;
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
      const float* src = held + (size_t)(j0 + col) * a.dim + i;
      if (VEC) {
        if (live && i < a.dim) s = *reinterpret_cast<const float4*>(src);
      } else if (live) {
        if (i < a.dim) s.x = src[0];
        if (i + 1 < a.dim) s.y = src[1];
        if (i + 2 < a.dim) s.z = src[2];
        if (i + 3 < a.dim) s.w = src[3];
      }
      S[col][2 * q] = pack2(s.x, s.y);
      S[col][2 * q + 1] = pack2(s.z, s.w);
    }

  // The read-outs of a tile wait as the lanes' own parts and are summed together: afterwards a lane holds the whole of one
  // token's, which it stores.
  const int out_tok = Fold::value_of(sub);
  const size_t out_stride = (size_t)a.heads * a.dim;
  float* out_at = a.out + (size_t)(first + out_tok) * out_stride + head * a.dim + j0;

  int round = 0;
  for (int tile = first; tile < end; tile += TILE, ++round) {
    const int count = min(TILE, end - tile), buffer = round & 1;
    const bool more = tile + TILE < end;
    if (more && tid == 0) stage_tile(tile + TILE, buffer ^ 1);  // its last readers passed the barrier below
    if (!__syncthreads_and(mbar_wait(&full[buffer], (round >> 1) & 1))) {
      if (tid == 0) {
        if (a.error) atomicExch(a.error, 6);
        mbar_wait(&full[buffer], (round >> 1) & 1);  // (bounded) no copy of its own in flight when the block leaves
        if (more) mbar_wait(&full[buffer ^ 1], ((round + 1) >> 1) & 1);
      }
      return;
    }
    const Stage& st = stages[buffer];
    float part[COLS][TILE];
#pragma unroll
    for (int tok = 0; tok < TILE; ++tok) {
      if (tok >= count) {
#pragma unroll
        for (int col = 0; col < COLS; ++col) part[col][tok] = 0.f;
        continue;
      }
      const float* piece = st.piece[tok];
      const float4 numbers = *reinterpret_cast<const float4*>(piece);
      const float* rows = piece + kDeltaNumbers + 4 * sub;
      const float* values = piece + kDeltaNumbers + 4 * KD + j0;  // (of columns past dim: zeros)
      Pair k[PER / 2], dot_k[COLS], dot_r[COLS];
#pragma unroll
      for (int col = 0; col < COLS; ++col) dot_k[col] = dot_r[col] = 0;
#pragma unroll
      for (int q = 0; q < PER / 4; ++q) {
        const ulonglong2 kv = *reinterpret_cast<const ulonglong2*>(rows + 4 * LANES * q);
        const ulonglong2 rv = *reinterpret_cast<const ulonglong2*>(rows + 3 * KD + 4 * LANES * q);
        k[2 * q] = kv.x;
        k[2 * q + 1] = kv.y;
#pragma unroll
        for (int col = 0; col < COLS; ++col) {
          dot_k[col] = fma2(kv.y, S[col][2 * q + 1], fma2(kv.x, S[col][2 * q], dot_k[col]));
          dot_r[col] = fma2(rv.y, S[col][2 * q + 1], fma2(rv.x, S[col][2 * q], dot_r[col]));
        }
      }
      float sum_k[COLS];
#pragma unroll
      for (int col = 0; col < COLS; ++col) {
        const float2 h = unpack2(dot_k[col]);
        sum_k[col] = h.x + h.y;
      }
#pragma unroll
      for (int offset = 1; offset < LANES; offset <<= 1)
#pragma unroll
        for (int col = 0; col < COLS; ++col) sum_k[col] += __shfl_xor_sync(0xffffffffu, sum_k[col], offset);
      Pair g2[COLS], v2[COLS];
#pragma unroll
      for (int col = 0; col < COLS; ++col) {
        const float g = -numbers.x * sum_k[col], v = values[col];
        const float2 h = unpack2(dot_r[col]);
        part[col][tok] = h.x + h.y + (sub == 0 ? v * numbers.y + g * numbers.z : 0.f);
        g2[col] = pack2(g, g);
        v2[col] = pack2(v, v);
      }
#pragma unroll
      for (int q = 0; q < PER / 4; ++q) {
        const ulonglong2 wv = *reinterpret_cast<const ulonglong2*>(rows + KD + 4 * LANES * q);
        const ulonglong2 av = *reinterpret_cast<const ulonglong2*>(rows + 2 * KD + 4 * LANES * q);
#pragma unroll
        for (int col = 0; col < COLS; ++col) {
          S[col][2 * q] = fma2(k[2 * q], fma2(av.x, g2[col], v2[col]), mul2(wv.x, S[col][2 * q]));
          S[col][2 * q + 1] = fma2(k[2 * q + 1], fma2(av.y, g2[col], v2[col]), mul2(wv.y, S[col][2 * q + 1]));
        }
      }
    }
#pragma unroll
    for (int col = 0; col < COLS; ++col) {
      const float o = Fold::run(part[col], sub);
      if (sub < TILE && out_tok < count && j0 + col < a.dim) out_at[col] = o;
    }
    out_at += TILE * out_stride;
    __syncthreads();  // everyone is done with this stage before the copies of the tile after next land in it
  }
#pragma unroll
  for (int col = 0; col < COLS; ++col) {
    if (j0 + col >= a.dim) continue;
#pragma unroll
    for (int p = 0; p < PER / 2; ++p) {
      const int i = 4 * sub + 4 * LANES * (p / 2) + 2 * (p % 2);
      const float2 s = unpack2(S[col][p]);
      float* dst = held + (size_t)(j0 + col) * a.dim + i;
      if (i < a.dim) dst[0] = s.x;
      if (i + 1 < a.dim) dst[1] = s.y;
    }
  }
}

template <int KD, int LANES, int COLS, int THREADS>
static cudaError_t launch_delta_as(const DeltaArgs& a, int num_seqs, bool vec, cudaStream_t stream) {
  constexpr int TILE = 8;
  constexpr int CB = THREADS / LANES * COLS;
  const dim3 grid(num_seqs, a.heads, (a.dim + CB - 1) / CB);
  const size_t shared = 2 * sizeof(DeltaStage<KD, TILE>);
  auto run = [&](auto kernel) {
    if (shared > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
    kernel<<<grid, THREADS, shared, stream>>>(a);
  };
  if (vec) run(channel_delta_kernel<KD, LANES, COLS, TILE, THREADS, true>);
  else run(channel_delta_kernel<KD, LANES, COLS, TILE, THREADS, false>);
  return cudaGetLastError();
}

template <int KD, int LANES, int COLS>
static cudaError_t launch_delta(const DeltaArgs& a, int num_seqs, bool vec, int threads, cudaStream_t stream) {
  if (threads >= 256) return launch_delta_as<KD, LANES, COLS, 256>(a, num_seqs, vec, stream);
  if (threads >= 128) return launch_delta_as<KD, LANES, COLS, 128>(a, num_seqs, vec, stream);
  return launch_delta_as<KD, LANES, COLS, 64>(a, num_seqs, vec, stream);
}

// lanes and columns of a thread as asked for, where a head has room for them.
template <int KD>
static cudaError_t dispatch_delta(const DeltaArgs& a, int num_seqs, bool vec, int lanes, int cols, int threads,
                                  cudaStream_t stream) {
  if constexpr (KD >= 128) {
    if (lanes == 32 && cols == 1) return launch_delta<KD, 32, 1>(a, num_seqs, vec, threads, stream);
    if (lanes == 32) return launch_delta<KD, 32, 2>(a, num_seqs, vec, threads, stream);
  }
  if constexpr (KD >= 64) {
    if (lanes >= 16 && cols == 1) return launch_delta<KD, 16, 1>(a, num_seqs, vec, threads, stream);
    if (lanes >= 16 && cols == 4) return launch_delta<KD, 16, 4>(a, num_seqs, vec, threads, stream);
    if (lanes >= 16) return launch_delta<KD, 16, 2>(a, num_seqs, vec, threads, stream);
  }
  if (cols >= 4) return launch_delta<KD, 8, 4>(a, num_seqs, vec, threads, stream);
  if (cols >= 2) return launch_delta<KD, 8, 2>(a, num_seqs, vec, threads, stream);
  return launch_delta<KD, 8, 1>(a, num_seqs, vec, threads, stream);
}

}  // namespace distie

using namespace distie;

// Floats of scratch for a step whose multi-token entries fill `num_tiles` tiles (0 tiles: none).
extern "C" long long distie_selective_scan_scratch_floats(int num_tiles, int states, int channels) {
  return (long long)num_tiles * channels * (states + 1);
}

// x [tokens, channels]; dt, gate [tokens, channels]; B, C [tokens, states], views of one projection (the same slices).
// Rows first_row .. first_row + rows - 1 of the batch are walked token by token; with num_tiles > 0 the tiles in `tiles`
// (int32 pairs: first token, length) take the three-launch form, with `scratch` from the function above.
extern "C" int distie_selective_scan(const float* x, int x_stride, const float* dt, int dt_stride, int dt_splits,
                                     long long dt_split_stride, const float* b, const float* c, int bc_stride,
                                     int bc_splits, long long bc_split_stride, const float* gate, int gate_stride,
                                     int gate_splits, long long gate_split_stride, const float* rates, const float* skip,
                                     const float* dt_bias, float* state, void* out, int out_stride, const int* seq_bounds,
                                     const int* seq_seat, const int* token_seq, const int* tiles, int num_tiles,
                                     float* scratch, int first_row, int rows, int channels, int states, int lanes,
                                     int dtype, cudaStream_t stream) {
  if (rows <= 0 && num_tiles <= 0) return 0;
  if (channels < 1 || states < 1 || dt_splits < 1 || bc_splits < 1 || gate_splits < 1 || rows < 0 || first_row < 0 || num_tiles < 0 ||
      rows > 65535 || num_tiles > 65535 || (num_tiles > 0 && (!tiles || !scratch || !token_seq)))
    return DISTIE_ERR_ARG;
  if (states > 256) return DISTIE_ERR_UNSUPPORTED;
  SelectArgs a;
  a.x = x; a.x_stride = x_stride;
  a.dt = Sliced{dt, dt_stride, dt_splits, dt_split_stride};
  a.B = Sliced{b, bc_stride, bc_splits, bc_split_stride};
  a.C = Sliced{c, bc_stride, bc_splits, bc_split_stride};
  a.gate = Sliced{gate, gate_stride, gate_splits, gate_split_stride};
  a.rates = rates; a.skip = skip; a.dt_bias = dt_bias; a.state = state; a.out_stride = out_stride;
  a.seq_bounds = seq_bounds; a.seq_seat = seq_seat; a.token_seq = token_seq; a.tiles = tiles;
  a.channels = channels; a.states = states; a.first_row = first_row; a.num_tiles = num_tiles;
  a.tile_state = scratch;
  a.tile_steps = scratch ? scratch + (size_t)num_tiles * states * channels : nullptr;
  cudaError_t err;
  if (dtype == DISTIE_BF16) err = dispatch_select(a, (__nv_bfloat16*)out, rows, num_tiles > 0, lanes, stream);
  else if (dtype == DISTIE_F32) err = dispatch_select(a, (float*)out, rows, num_tiles > 0, lanes, stream);
  else return DISTIE_ERR_UNSUPPORTED;
  return err == cudaSuccess ? 0 : (int)err;
}

static int delta_width(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }

// Floats of scratch of the delta rule below.
extern "C" long long distie_channel_delta_scratch_floats(int tokens, int heads, int dim) {
  return (long long)tokens * heads * (kDeltaNumbers + (long long)kDeltaRows * delta_width(dim));
}

// proj [tokens, 4 heads dim (+ more)] = [r | k | v | rate], decay [tokens, heads dim] (each a matrix or slices); out
// [tokens, heads dim]; scratch 16-byte aligned.  lanes: threads that share a column (8, 16, 32), cols: columns of a thread.
extern "C" int distie_channel_delta(const float* proj, int proj_stride, int proj_splits, long long proj_split_stride,
                                    const float* decay, int decay_stride, int decay_splits, long long decay_split_stride,
                                    const float* decay_bias, const float* rate_bias, float* state, float* out,
                                    float* scratch, const int* seq_bounds, const int* seq_seat, int tokens, int num_seqs,
                                    int heads, int dim, int lanes, int cols, int threads, int* error,
                                    cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (heads < 1 || heads > 65535 || dim < 1 || num_seqs < 1 || proj_splits < 1 || decay_splits < 1 || !scratch || !state ||
      ((uintptr_t)scratch & 15))
    return DISTIE_ERR_ARG;
  if (dim > 256) return DISTIE_ERR_UNSUPPORTED;
  DeltaArgs a;
  a.proj = Sliced{proj, proj_stride, proj_splits, proj_split_stride};
  a.decay = Sliced{decay, decay_stride, decay_splits, decay_split_stride};
  a.decay_bias = decay_bias; a.rate_bias = rate_bias;
  a.scratch = scratch; a.width = delta_width(dim); a.error = error;
  a.state = state; a.out = out; a.seq_bounds = seq_bounds; a.seq_seat = seq_seat;
  a.tokens = tokens; a.heads = heads; a.dim = dim;
  channel_delta_prepare_kernel<<<dim3(tokens, tokens < 512 ? (heads + 3) / 4 : 1), 128, 0, stream>>>(a);
  DISTIE_LAUNCH_CHECK();
  const bool vec = dim % 4 == 0 && ((uintptr_t)state & 15) == 0;
  cudaError_t err;
  if (dim <= 32) err = dispatch_delta<32>(a, num_seqs, vec, lanes, cols, threads, stream);
  else if (dim <= 64) err = dispatch_delta<64>(a, num_seqs, vec, lanes, cols, threads, stream);
  else if (dim <= 128) err = dispatch_delta<128>(a, num_seqs, vec, lanes, cols, threads, stream);
  else err = dispatch_delta<256>(a, num_seqs, vec, lanes, cols, threads, stream);
  return err == cudaSuccess ? 0 : (int)err;
}
