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
// blocks compute a neighbour's h again instead of waiting for it: a block of the shifted form owns one token and computes
// the h of the token before it as well (the reads are the neighbour's, a moment apart: the L2 serves one of the two). The
// block with a sequence's first token of the step reads the state row and, at the end, writes it: with its own h, or, where
// the sequence goes on in other blocks, with the last token's h computed once more. So a row of state has one reader and
// writer, whatever the cut, and the value has the bits that any other block would have given it.
//
// `x_stream` is the distance between a token's streams; 0 lets one row stand for all of them (they start out equal).
#include <math.h>

#include "common.cuh"

namespace {
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

// One token by all threads of the block: thread i owns channel pieces i, i + blockDim, ... (NP of them at most), gets its
// channels of u and returns their sum of squares. S: the number of streams, 0 for any number (then x is read once per
// stream that is made).
template <typename T, int S, int C, int NP>
__device__ __forceinline__ float token_sum(const StreamProblem& p, const float* small, size_t token, bool write, float (&h)[NP][C]) {
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
  return ss;
}

// u to h, in place, from the block's sum of squares.
template <int C, int NP>
__device__ __forceinline__ void token_norm(const StreamProblem& p, float ss, float (&h)[NP][C]) {
  const float inv = 1.0f / sqrtf(ss / (float)p.width + p.eps);
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

// `block_sum` of two values at once, each in the order of `block_sum` (so either has the bits it would have alone).
__device__ __forceinline__ float2 block_sum_pair(float a, float b, float2* scratch /* >= 33 */) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();
  if (lane == 0) scratch[warp] = make_float2(a, b);
  __syncthreads();
  if (threadIdx.x == 0) {
    float2 total = make_float2(0.f, 0.f);
    for (int w = 0; w < nwarps; ++w) {
      total.x += scratch[w].x;
      total.y += scratch[w].y;
    }
    scratch[32] = total;
  }
  __syncthreads();
  return scratch[32];
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
  const float ss = token_sum<T, S, C, NP>(p, small, token, true, h);
  token_norm<C, NP>(p, block_sum(ss, scratch), h);
  T* o = out + (size_t)blockIdx.x * p.width;
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * C;
    if (c < p.width) Channels<T, C>::store(o + c, h[k]);
  }
}

// A block per token. The token's h and the h of the token before it are made side by side: their loads are in flight
// together and their sums meet in one reduction. Whether the token is a sequence's first of the step is looked up in cu_q.
// The step's descriptors are older than every kernel of the step (the copy that brings them is no kernel, so nothing
// overtakes it) and a state row is written by this kernel of an earlier step only, so both are read before the wait.
template <typename T, int S, int C, int NP>
__global__ void __launch_bounds__(MAX_THREADS)
stream_norm_shift_kernel(const StreamProblem p, T* __restrict__ out, const float* __restrict__ mu, float* __restrict__ state,
                         long state_stride, const int* __restrict__ cu_q, const int* __restrict__ state_slots, int n_seqs) {
  __shared__ float small[MAX_STREAMS * MAX_STREAMS + 2 * MAX_STREAMS];
  __shared__ float2 scratch[33];
  __shared__ int first_of;      // the sequence that starts here, or -1
  pdl_launch_dependents();
  const size_t token = blockIdx.x;
  if (threadIdx.x == 0) first_of = -1;
  __syncthreads();
  for (int i = threadIdx.x; i < n_seqs; i += blockDim.x)
    if (cu_q[i] == (int)token) first_of = i;      // no sequence of a step is empty: at most one
  load_small(p, small);
  const int seq = first_of;
  float before[NP][C], h[NP][C];
  float* row = nullptr;
  if (seq >= 0) {
    row = state + (size_t)state_slots[seq] * state_stride;
#pragma unroll
    for (int k = 0; k < NP; ++k) {
      const int c = (threadIdx.x + k * blockDim.x) * C;
      if (c < p.width) Channels<float, C>::load(row + c, before[k]);
    }
  }
  pdl_wait();
  float ss_before = 0.f;
  if (!row) ss_before = token_sum<T, S, C, NP>(p, small, token - 1, false, before);
  const float ss = token_sum<T, S, C, NP>(p, small, token, true, h);
  const float2 sums = block_sum_pair(ss, ss_before, scratch);
  token_norm<C, NP>(p, sums.x, h);
  if (!row) token_norm<C, NP>(p, sums.y, before);
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * C;
    if (c < p.width) {
      float m[C], v[C];
      Channels<float, C>::load(mu + c, m);
#pragma unroll
      for (int i = 0; i < C; ++i) v[i] = fmaf(before[k][i] - h[k][i], m[i], h[k][i]);
      Channels<T, C>::store(out + token * p.width + c, v);
    }
  }
  if (!row) return;
  const size_t end = (size_t)cu_q[seq + 1] - 1;
  if (end != token) {     // the sequence goes on in other blocks: its last token's h once more, for the state row
    const float last = token_sum<T, S, C, NP>(p, small, end, false, h);
    token_norm<C, NP>(p, block_sum_pair(last, 0.f, scratch).x, h);
  }
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int c = (threadIdx.x + k * blockDim.x) * C;
    if (c < p.width) Channels<float, C>::store(row + c, h[k]);
  }
}

struct ShiftArguments {
  const float* mu;
  float* state;
  long state_stride;
  const int *cu_q, *state_slots;
  int n_seqs;
};

template <typename T, int S, int C, int NP>
int launch_streams(const StreamProblem& p, void* out, const int* rows, int blocks, int threads, const ShiftArguments& sh, cudaStream_t stream) {
  if (sh.mu)
    lb_launch(stream_norm_shift_kernel<T, S, C, NP>, blocks, threads, 0, stream, p, (T*)out, sh.mu, sh.state, sh.state_stride, sh.cu_q,
              sh.state_slots, sh.n_seqs);
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
  const int threads = pieces <= 256 ? 128 : (pieces <= 512 ? 256 : MAX_THREADS);
  const bool two = pieces <= 2 * threads;         // pieces a thread: at most two, or at most four
  switch (p.streams) {
    case 2: return two ? launch_streams<T, 2, 4, 2>(p, out, rows, blocks, threads, sh, stream)
                       : launch_streams<T, 2, 4, 4>(p, out, rows, blocks, threads, sh, stream);
    case 4: return two ? launch_streams<T, 4, 4, 2>(p, out, rows, blocks, threads, sh, stream)
                       : launch_streams<T, 4, 4, 4>(p, out, rows, blocks, threads, sh, stream);
    default: return launch_streams<T, 0, 4, 4>(p, out, rows, blocks, threads, sh, stream);
  }
}
}  // namespace

LB_EXPORT int lb_stream_max() { return MAX_STREAMS; }

// x float [tokens, streams, width] by strides; y [tokens, width] of `dtype` or null (then mix and gain are null too);
// mix float [streams, streams] ([from, to]), gain, read float [streams] (read null: ones); x_out float [tokens, streams,
// width] or null, never the buffer of x; out [blocks, width] of `dtype`. mu null: a block per token, or per entry of
// `rows` (then x_out is null). mu float [width]: the shifted form, `blocks` tokens in `n_seqs` sequences (cu_q [n_seqs + 1]:
// their first tokens), a state row of `state_stride` floats per slot.
LB_EXPORT int lb_stream_norm(int dtype, const float* x, long x_token, long x_stream, const void* y, const float* mix,
                             const float* gain, const float* read, float* x_out, const float* weight, float eps, void* out,
                             const int* rows, int blocks, int width, int streams, const float* mu, float* state,
                             long state_stride, const int* cu_q, const int* state_slots, int n_seqs, cudaStream_t stream) {
  if (blocks <= 0) return 0;
  if (width <= 0 || streams < 1 || streams > MAX_STREAMS || !x || !weight || !out || (y && (!mix || !gain)) || (rows && x_out) ||
      (x_out && x_out == x) || (mu && (rows || !state || !cu_q || !state_slots || n_seqs < 1)))
    return LB_ERR_SIZE;
  const StreamProblem p{x, x_token, x_stream, y, mix, gain, read, x_out, weight, eps, width, streams};
  const ShiftArguments sh{mu, state, state_stride, cu_q, state_slots, n_seqs};
  const bool vec = width % 4 == 0 && x_token % 4 == 0 && x_stream % 4 == 0 && state_stride % 4 == 0 &&
                   ((uintptr_t)x | (uintptr_t)y | (uintptr_t)x_out | (uintptr_t)weight | (uintptr_t)out | (uintptr_t)mu |
                    (uintptr_t)state) % 16 == 0;
  if (dtype == LB_F32) return dispatch_streams<float>(p, out, rows, blocks, vec, sh, stream);
  if (dtype == LB_BF16) return dispatch_streams<bf16>(p, out, rows, blocks, vec, sh, stream);
  return LB_ERR_DTYPE;
}
