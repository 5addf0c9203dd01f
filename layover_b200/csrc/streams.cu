// Several residual streams instead of one: what happens between two sub-layers, as ONE kernel. Per token, with the
// streams x_1 .. x_S (32-bit whatever the run's type T), the output y of the sub-layer before and its small matrices,
//
//   x'_t = sum_s mix[s, t] x_s + gain[t] y            (all streams at once from the old ones; y null: x' = x)
//   u    = sum_t read[t] x'_t                         (read null: the plain sum)
//   h    = u * rsqrt(mean(u^2) + eps) * weight
//   out  = T(h)                                       or, with a token shift, T(h + (h_before - h) * mu)
//
// h_before is the h of the sequence's previous token, unrounded and 32-bit: zeros before the first token, for a step's
// first token the request's state row. Everything is 32-bit arithmetic in a fixed order, rounded once at the store.
//
// The streams are written to another buffer than they are read from (x_out null: not written at all), which is what lets
// blocks compute a neighbour's h again instead of waiting for it: a block of the shifted form owns SHIFT_TOKENS tokens of
// one sequence and first computes the h of the token before them. The block with a sequence's first token of the step
// reads the state row and, at the end, writes it: with its own last token's h, or, where the sequence goes on in other
// blocks, with the last token's h computed once more. So a row of state has one reader and writer, whatever the cut,
// and the value has the bits that any other block would have given it.
//
// `x_stream` is the distance between a token's streams; 0 lets one row stand for all of them (they start out equal).
#include <math.h>

#include "common.cuh"

namespace {
constexpr int SHIFT_TOKENS = 4;
constexpr int MAX_STREAMS = 16;
constexpr int MAX_THREADS = 512;      // so widths up to 8192 (4096 where they are no multiple of 4)

// C neighbouring channels of a row at once.
template <typename T, int C> struct Channels;
template <typename T> struct Channels<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = Elem<T>::load(p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { Elem<T>::store(p, v[0]); }
};
template <> struct Channels<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct Channels<bf16, 4> {
  static __device__ __forceinline__ void load(const bf16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    v[0] = __low2float(lo); v[1] = __high2float(lo); v[2] = __low2float(hi); v[3] = __high2float(hi);
  }
  static __device__ __forceinline__ void store(bf16* p, const float (&v)[4]) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&lo);
    raw.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
  }
};

struct StreamProblem {
  const float* x;
  long x_token, x_stream;
  const void* y;
  const float *mix, *gain, *read;
  float* x_out;
  const float* weight;
  float eps;
  int width, streams;
};

// One token by all threads of the block: thread i owns channel pieces i, i + blockDim, ... (NP of them at most) and gets
// its channels of h. S: the number of streams, 0 for any number (then x is read once per stream that is made).
template <typename T, int S, int C, int NP>
__device__ __forceinline__ void token_norm(const StreamProblem& p, const float* small, size_t token, bool write, float* scratch,
                                           float (&h)[NP][C]) {
  const int streams = S ? S : p.streams;
  const float *mix = small, *gain = small + streams * streams, *read = gain + streams;
  const float* xr = p.x + token * p.x_token;
  const T* yr = p.y ? (const T*)p.y + token * p.width : nullptr;
  float* xo = p.x_out && write ? p.x_out + token * streams * p.width : nullptr;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * C;
#pragma unroll
    for (int i = 0; i < C; ++i) h[k][i] = 0.f;
    if (c < p.width) {
      float y[C];
      if (yr) Channels<T, C>::load(yr + c, y);
      if (S) {
        float x[S ? S : 1][C];
#pragma unroll
        for (int s = 0; s < S; ++s) Channels<float, C>::load(xr + s * p.x_stream + c, x[s]);
#pragma unroll
        for (int t = 0; t < S; ++t) {
          float v[C];
#pragma unroll
          for (int i = 0; i < C; ++i) {
            v[i] = x[t][i];
            if (yr) {
              v[i] = 0.f;
#pragma unroll
              for (int s = 0; s < S; ++s) v[i] = fmaf(mix[s * S + t], x[s][i], v[i]);
              v[i] = fmaf(gain[t], y[i], v[i]);
            }
            h[k][i] = fmaf(read[t], v[i], h[k][i]);
          }
          if (xo) Channels<float, C>::store(xo + (size_t)t * p.width + c, v);
        }
      } else {
        for (int t = 0; t < streams; ++t) {
          float v[C];
          if (yr) {
#pragma unroll
            for (int i = 0; i < C; ++i) v[i] = 0.f;
            for (int s = 0; s < streams; ++s) {
              float x[C];
              Channels<float, C>::load(xr + s * p.x_stream + c, x);
#pragma unroll
              for (int i = 0; i < C; ++i) v[i] = fmaf(mix[s * streams + t], x[i], v[i]);
            }
#pragma unroll
            for (int i = 0; i < C; ++i) v[i] = fmaf(gain[t], y[i], v[i]);
          } else {
            Channels<float, C>::load(xr + t * p.x_stream + c, v);
          }
#pragma unroll
          for (int i = 0; i < C; ++i) h[k][i] = fmaf(read[t], v[i], h[k][i]);
          if (xo) Channels<float, C>::store(xo + (size_t)t * p.width + c, v);
        }
      }
#pragma unroll
      for (int i = 0; i < C; ++i) ss = fmaf(h[k][i], h[k][i], ss);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * C;
    if (c < p.width) {
      float w[C];
      Channels<float, C>::load(p.weight + c, w);
#pragma unroll
      for (int i = 0; i < C; ++i) h[k][i] = h[k][i] * inv * w[i];
    }
  }
}

// The small matrices into shared memory: they are weights, which no kernel writes, so this may run before the wait.
__device__ __forceinline__ void load_small(const StreamProblem& p, float* small) {
  const int S = p.streams, total = S * S + 2 * S;
  for (int i = threadIdx.x; i < total; i += blockDim.x) {
    float v = 1.f;
    if (i < S * S) v = p.mix ? p.mix[i] : 0.f;
    else if (i < S * S + S) v = p.gain ? p.gain[i - S * S] : 0.f;
    else if (p.read) v = p.read[i - S * S - S];
    small[i] = v;
  }
  __syncthreads();
}

// A block per token (with `rows`: per listed token).
template <typename T, int S, int C, int NP>
__global__ void __launch_bounds__(MAX_THREADS)
stream_norm_kernel(const StreamProblem p, T* __restrict__ out, const int* __restrict__ rows) {
  __shared__ float small[MAX_STREAMS * MAX_STREAMS + 2 * MAX_STREAMS];
  __shared__ float scratch[33];
  pdl_launch_dependents();
  load_small(p, small);
  pdl_wait();
  const size_t token = rows ? (size_t)rows[blockIdx.x] : (size_t)blockIdx.x;
  float h[NP][C];
  token_norm<T, S, C, NP>(p, small, token, true, scratch, h);
  T* o = out + (size_t)blockIdx.x * p.width;
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * C;
    if (c < p.width) Channels<T, C>::store(o + c, h[k]);
  }
}

// A block per tile of SHIFT_TOKENS tokens of one sequence (the tile lists name the sequence and the tile's first token).
template <typename T, int S, int C, int NP>
__global__ void __launch_bounds__(MAX_THREADS)
stream_norm_shift_kernel(const StreamProblem p, T* __restrict__ out, const float* __restrict__ mu, float* __restrict__ state,
                         long state_stride, const int* __restrict__ cu_q, const int* __restrict__ state_slots,
                         const int* __restrict__ tile_seq, const int* __restrict__ tile_q0) {
  __shared__ float small[MAX_STREAMS * MAX_STREAMS + 2 * MAX_STREAMS];
  __shared__ float scratch[33];
  pdl_launch_dependents();
  load_small(p, small);
  pdl_wait();
  const int seq = tile_seq[blockIdx.x], at = tile_q0[blockIdx.x];
  const size_t row0 = (size_t)cu_q[seq];
  const int length = cu_q[seq + 1] - (int)row0, n = min(SHIFT_TOKENS, length - at);
  if (n <= 0) return;
  float* row = state + (size_t)state_slots[seq] * state_stride;
  float before[NP][C], h[NP][C];
  if (at == 0) {
#pragma unroll
    for (int k = 0; k < NP; ++k) {
      const int c = (threadIdx.x + k * blockDim.x) * C;
      if (c < p.width) Channels<float, C>::load(row + c, before[k]);
    }
  }
  // the token before the tile (not with the state row in its place), the tile's own, and, for the state row of a sequence
  // that goes on in other blocks, its last token
  const int end = at == 0 && length > n ? n + 1 : n;
  for (int j = at > 0 ? -1 : 0; j < end; ++j) {
    const bool own = j >= 0 && j < n;
    const size_t token = row0 + (j < n ? at + j : length - 1);
    token_norm<T, S, C, NP>(p, small, token, own, scratch, h);
#pragma unroll
    for (int k = 0; k < NP; ++k) {
      const int c = (threadIdx.x + k * blockDim.x) * C;
      if (own && c < p.width) {
        float m[C], v[C];
        Channels<float, C>::load(mu + c, m);
#pragma unroll
        for (int i = 0; i < C; ++i) v[i] = fmaf(before[k][i] - h[k][i], m[i], h[k][i]);
        Channels<T, C>::store(out + token * p.width + c, v);
      }
#pragma unroll
      for (int i = 0; i < C; ++i) before[k][i] = h[k][i];
    }
  }
  if (at > 0) return;
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * C;
    if (c < p.width) Channels<float, C>::store(row + c, before[k]);
  }
}

struct ShiftArguments {
  const float* mu;
  float* state;
  long state_stride;
  const int *cu_q, *state_slots, *tile_seq, *tile_q0;
};

template <typename T, int S, int C, int NP>
int launch_streams(const StreamProblem& p, void* out, const int* rows, int blocks, int threads, const ShiftArguments& sh, cudaStream_t stream) {
  if (sh.mu)
    lb_launch(stream_norm_shift_kernel<T, S, C, NP>, blocks, threads, 0, stream, p, (T*)out, sh.mu, sh.state, sh.state_stride, sh.cu_q,
              sh.state_slots, sh.tile_seq, sh.tile_q0);
  else
    lb_launch(stream_norm_kernel<T, S, C, NP>, blocks, threads, 0, stream, p, (T*)out, rows);
  return lb_last_error();
}

template <typename T>
int dispatch_streams(const StreamProblem& p, void* out, const int* rows, int blocks, bool vec, const ShiftArguments& sh, cudaStream_t stream) {
  // form and block size depend on the width and the buffers' alignment only, never on the batch
  if (!vec) {
    if (p.width > 8 * MAX_THREADS) return LB_ERR_SIZE;
    return launch_streams<T, 0, 1, 8>(p, out, rows, blocks, p.width <= 1024 ? 128 : MAX_THREADS, sh, stream);
  }
  const int pieces = p.width / 4;
  if (pieces > 4 * MAX_THREADS) return LB_ERR_SIZE;
  const int threads = pieces <= 256 ? 128 : (pieces <= 1024 ? 256 : MAX_THREADS);
  switch (p.streams) {
    case 2: return launch_streams<T, 2, 4, 4>(p, out, rows, blocks, threads, sh, stream);
    case 4: return launch_streams<T, 4, 4, 4>(p, out, rows, blocks, threads, sh, stream);
    default: return launch_streams<T, 0, 4, 4>(p, out, rows, blocks, threads, sh, stream);
  }
}
}  // namespace

LB_EXPORT int lb_stream_shift_tokens() { return SHIFT_TOKENS; }
LB_EXPORT int lb_stream_max() { return MAX_STREAMS; }

// x float [tokens, streams, width] by strides; y [tokens, width] of `dtype` or null (then mix and gain are null too);
// mix float [streams, streams] ([from, to]), gain, read float [streams] (read null: ones); x_out float [tokens, streams,
// width] or null, never the buffer of x; out [blocks, width] of `dtype`. mu null: a block per token, or per entry of
// `rows` (then x_out is null). mu float [width]: the shifted form, `blocks` tiles, state rows of `state_stride` floats.
LB_EXPORT int lb_stream_norm(int dtype, const float* x, long x_token, long x_stream, const void* y, const float* mix,
                             const float* gain, const float* read, float* x_out, const float* weight, float eps, void* out,
                             const int* rows, int blocks, int width, int streams, const float* mu, float* state,
                             long state_stride, const int* cu_q, const int* state_slots, const int* tile_seq,
                             const int* tile_q0, cudaStream_t stream) {
  if (blocks <= 0) return 0;
  if (width <= 0 || streams < 1 || streams > MAX_STREAMS || !x || !weight || !out || (y && (!mix || !gain)) || (rows && x_out) ||
      (x_out && x_out == x) || (mu && (rows || !state || !cu_q || !state_slots || !tile_seq || !tile_q0)))
    return LB_ERR_SIZE;
  const StreamProblem p{x, x_token, x_stream, y, mix, gain, read, x_out, weight, eps, width, streams};
  const ShiftArguments sh{mu, state, state_stride, cu_q, state_slots, tile_seq, tile_q0};
  const bool vec = width % 4 == 0 && x_token % 4 == 0 && x_stream % 4 == 0 && state_stride % 4 == 0 &&
                   ((uintptr_t)x | (uintptr_t)y | (uintptr_t)x_out | (uintptr_t)weight | (uintptr_t)out | (uintptr_t)mu |
                    (uintptr_t)state) % 16 == 0;
  if (dtype == LB_F32) return dispatch_streams<float>(p, out, rows, blocks, vec, sh, stream);
  if (dtype == LB_BF16) return dispatch_streams<bf16>(p, out, rows, blocks, vec, sh, stream);
  return LB_ERR_DTYPE;
}
