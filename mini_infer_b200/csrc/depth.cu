// Around a layer whose norms stand behind its branches: the norm and the sum behind a branch, the average
// over the results of all layers so far, and the short causal convolution in front of the next mixer.
//
//   mi_branch_depth   per token (row), fp32:
//                       X = stream + ((y - mean) * rstd * w + b)        (without a branch: X = stream)
//                       x = X, or, with `avg`, sum_{j < n_prev} a[j] X_j + a[n_prev] X with X_0 = first
//                           and X_(j+1) = results[j] (fp32 [n_prev - 1 and more][M][H])
//                       and, with `conv_w` (steps of one token per request), the convolution of mi_input_conv
//                       on x, whose earlier inputs are the request's state, which moves on by one token.
//                     Outputs, each optional: X (stream_out; may be the stream itself, or a slot of
//                     `results`), x (avg_out), x in the compute dtype (copy), the convolved row (conv_out).
//   mi_input_conv     per channel  out_t = h_t + sum_j w[j] h_(t - taps + 1 + j)  over a request's portion, the
//                     inputs before the portion coming from the request's state ([taps - 1][H] fp32, oldest
//                     first), which then holds the portion's last taps - 1 inputs.
//
// Mean and variance are fp32, the variance is the mean of the squared deviations.  One block per row;
// gains and biases fp32.  Every sum runs in an order that depends on H (and n_prev, taps) alone, and both
// convolutions add up in the same order, so a row's bits do not depend on how the work was cut.
#include "common.cuh"

MI_DEFINE_ERROR_API()

#define MAX_TAPS 16

// V neighbouring elements (4 where sizes and alignment allow, else 1)
template <typename T, int V>
struct Pack;
template <typename T>
struct Pack<T, 4> {
  static __device__ __forceinline__ void load(const T* p, float (&f)[4]) {
    Vec4<T> v;
    v.load(p);
    v.get(f);
  }
  static __device__ __forceinline__ void store(T* p, const float (&f)[4]) {
    Vec4<T> v;
    v.set(f);
    v.store(p);
  }
};
template <typename T>
struct Pack<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&f)[1]) { f[0] = mi_to_float(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&f)[1]) { *p = mi_from_float<T>(f[0]); }
};

struct BranchDepthArgs {
  const float* stream;
  const void* branch;      // T [M, branch_stride], or null
  int branch_stride;
  const float *w, *b;
  float eps;
  float* stream_out;
  void* copy;              // T [M, H]
  const float* first;      // X_0 [M, H]
  const float* results;    // X_1 ...: [n_prev - 1][M][H]
  int n_prev;              // earlier results, X_0 included; 0: no average
  const float* avg;        // [n_prev + 1]
  float* avg_out;
  const float* conv_w;     // [taps][H], or null
  int taps;
  float* conv_state;       // [slots][conv_stride]: [taps - 1][H] per slot
  long long conv_stride;
  const int* state_slot;   // [M]
  void* conv_out;          // T [M, H]
  int M, H;
};

template <typename T, int V>
__global__ void branch_depth_kernel(const BranchDepthArgs a) {
  mi_pdl_launch_dependents();
  extern __shared__ __align__(16) float row[];       // [H] the branch's row (nothing without a branch)
  __shared__ float red[32];
  const int t = blockIdx.x, H = a.H;
  mi_pdl_wait();
  const size_t at = (size_t)t * H;
  float mean = 0.f, rstd = 0.f;
  if (a.branch) {
    const T* y = reinterpret_cast<const T*>(a.branch) + (size_t)t * a.branch_stride;
    float sum = 0.f;
    for (int k = V * threadIdx.x; k < H; k += V * blockDim.x) {
      float f[V];
      Pack<T, V>::load(y + k, f);
      Pack<float, V>::store(row + k, f);
#pragma unroll
      for (int i = 0; i < V; ++i) sum += f[i];
    }
    mean = mi_block_sum(sum, red) / (float)H;
    float sq = 0.f;
    for (int k = V * threadIdx.x; k < H; k += V * blockDim.x) {      // each thread reads what it wrote
      float f[V];
      Pack<float, V>::load(row + k, f);
#pragma unroll
      for (int i = 0; i < V; ++i) sq += (f[i] - mean) * (f[i] - mean);
    }
    rstd = 1.f / sqrtf(mi_block_sum(sq, red) / (float)H + a.eps);
  }
  float* tail = a.conv_w && a.taps > 1 ? a.conv_state + (size_t)a.state_slot[t] * a.conv_stride : nullptr;
  for (int k = V * threadIdx.x; k < H; k += V * blockDim.x) {
    float x[V];
    Pack<float, V>::load(a.stream + at + k, x);
    if (a.branch) {
      float f[V], g[V], c[V];
      Pack<float, V>::load(row + k, f);
      Pack<float, V>::load(a.w + k, g);
      Pack<float, V>::load(a.b + k, c);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] += (f[i] - mean) * rstd * g[i] + c[i];
    }
    if (a.stream_out) Pack<float, V>::store(a.stream_out + at + k, x);
    if (a.n_prev > 0) {
      float acc[V], f[V];
      Pack<float, V>::load(a.first + at + k, f);
      const float a0 = a.avg[0], an = a.avg[a.n_prev];
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = a0 * f[i];
      const float* res = a.results + at + k;
      const size_t pitch = (size_t)a.M * H;
      int j = 1;
      for (; j + 4 <= a.n_prev; j += 4) {             // four results in flight; added in order
        float r[4][V];
#pragma unroll
        for (int u = 0; u < 4; ++u) Pack<float, V>::load(res + (size_t)(j - 1 + u) * pitch, r[u]);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float wj = a.avg[j + u];
#pragma unroll
          for (int i = 0; i < V; ++i) acc[i] = fmaf(wj, r[u][i], acc[i]);
        }
      }
      for (; j < a.n_prev; ++j) {
        Pack<float, V>::load(res + (size_t)(j - 1) * pitch, f);
        const float wj = a.avg[j];
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(wj, f[i], acc[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] = fmaf(an, x[i], acc[i]);
      if (a.avg_out) Pack<float, V>::store(a.avg_out + at + k, x);
    }
    if (a.copy) Pack<T, V>::store(reinterpret_cast<T*>(a.copy) + at + k, x);
    if (a.conv_w) {
      float acc[V], w[V], in[V];
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = 0.f;
      for (int j = 0; j < a.taps - 1; ++j) {
        Pack<float, V>::load(a.conv_w + (size_t)j * H + k, w);
        Pack<float, V>::load(tail + (size_t)j * H + k, in);
        if (j > 0) Pack<float, V>::store(tail + (size_t)(j - 1) * H + k, in);    // the state moves on by one token
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(w[i], in[i], acc[i]);
      }
      Pack<float, V>::load(a.conv_w + (size_t)(a.taps - 1) * H + k, w);
      if (a.taps > 1) Pack<float, V>::store(tail + (size_t)(a.taps - 2) * H + k, x);
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = x[i] + fmaf(w[i], x[i], acc[i]);
      Pack<T, V>::store(reinterpret_cast<T*>(a.conv_out) + at + k, acc);
    }
  }
}

// The same for rows of up to 4096 channels in whole 16-byte pieces: a thread holds four channels from the first
// load to the last store, and everything that does not depend on the row's statistics is asked for before them.
#define ROW_MAX_THREADS 1024
// AVG, CONV: whether the launch averages and convolves (an instance without them needs half the registers).
template <typename T, bool AVG, bool CONV>
__global__ void __launch_bounds__(ROW_MAX_THREADS)
branch_depth_row_kernel(const BranchDepthArgs a) {
  mi_pdl_launch_dependents();
  __shared__ float red[32];
  const int t = blockIdx.x, H = a.H, k = 4 * threadIdx.x;
  const bool on = k < H;
  const size_t at = (size_t)t * H + k;
  float g[4] = {}, c[4] = {}, y[4] = {}, x[4] = {}, acc[4] = {};
  if (on && a.branch) {                // immutable: may be read before the kernels in front have finished
    Pack<float, 4>::load(a.w + k, g);
    Pack<float, 4>::load(a.b + k, c);
  }
  mi_pdl_wait();
  if (on) {
    if (a.branch) Pack<T, 4>::load(reinterpret_cast<const T*>(a.branch) + (size_t)t * a.branch_stride + k, y);
    Pack<float, 4>::load(a.stream + at, x);
    if (AVG) {
      float f[4];
      Pack<float, 4>::load(a.first + at, f);
      const float a0 = a.avg[0];
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i] = a0 * f[i];
      const float* res = a.results + at;
      const size_t pitch = (size_t)a.M * H;
      int j = 1;
      for (; j + 4 <= a.n_prev; j += 4) {             // four results in flight; added in order
        float r[4][4];
#pragma unroll
        for (int u = 0; u < 4; ++u) Pack<float, 4>::load(res + (size_t)(j - 1 + u) * pitch, r[u]);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float wj = a.avg[j + u];
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[i] = fmaf(wj, r[u][i], acc[i]);
        }
      }
      for (; j < a.n_prev; ++j) {
        Pack<float, 4>::load(res + (size_t)(j - 1) * pitch, f);
        const float wj = a.avg[j];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i] = fmaf(wj, f[i], acc[i]);
      }
    }
  }
  if (a.branch) {
    const float mean = mi_block_sum((y[0] + y[1]) + (y[2] + y[3]), red) / (float)H;
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      y[i] -= mean;
      sq += y[i] * y[i];
    }
    const float rstd = 1.f / sqrtf(mi_block_sum(on ? sq : 0.f, red) / (float)H + a.eps);
#pragma unroll
    for (int i = 0; i < 4; ++i) x[i] += y[i] * rstd * g[i] + c[i];
  }
  if (!on) return;
  if (a.stream_out) Pack<float, 4>::store(a.stream_out + at, x);
  if (AVG) {
    const float an = a.avg[a.n_prev];
#pragma unroll
    for (int i = 0; i < 4; ++i) x[i] = fmaf(an, x[i], acc[i]);
    if (a.avg_out) Pack<float, 4>::store(a.avg_out + at, x);
  }
  if (a.copy) Pack<T, 4>::store(reinterpret_cast<T*>(a.copy) + at, x);
  if (CONV) {
    float* tail = a.taps > 1 ? a.conv_state + (size_t)a.state_slot[t] * a.conv_stride + k : nullptr;
    float s[4] = {}, w[4], in[4];
    for (int j = 0; j < a.taps - 1; ++j) {
      Pack<float, 4>::load(a.conv_w + (size_t)j * H + k, w);
      Pack<float, 4>::load(tail + (size_t)j * H, in);
      if (j > 0) Pack<float, 4>::store(tail + (size_t)(j - 1) * H, in);     // the state moves on by one token
#pragma unroll
      for (int i = 0; i < 4; ++i) s[i] = fmaf(w[i], in[i], s[i]);
    }
    Pack<float, 4>::load(a.conv_w + (size_t)(a.taps - 1) * H + k, w);
    if (a.taps > 1) Pack<float, 4>::store(tail + (size_t)(a.taps - 2) * H, x);
#pragma unroll
    for (int i = 0; i < 4; ++i) s[i] = x[i] + fmaf(w[i], x[i], s[i]);
    Pack<T, 4>::store(reinterpret_cast<T*>(a.conv_out) + at, s);
  }
}

extern "C" int mi_branch_depth(const float* stream, const void* branch, int branch_stride, const float* w,
                               const float* b, float eps, float* stream_out, void* copy, const float* first,
                               const float* results, int n_prev, const float* avg, float* avg_out,
                               const float* conv_w, int taps, float* conv_state, long long conv_stride,
                               const int* state_slot, void* conv_out, int M, int H, int dtype, cudaStream_t cu_stream) {
  if (M <= 0) return 0;
  if (H <= 0) MI_REFUSE("branch_depth: bad width %d", H);
  if (!stream || (branch && (!w || !b))) MI_REFUSE("branch_depth: a stream, and a branch with its gain and bias");
  if (n_prev < 0 || (n_prev > 0 && (!first || !avg || (n_prev > 1 && !results))))
    MI_REFUSE("branch_depth: an average over %d earlier results needs them and their weights", n_prev);
  if (conv_w && (taps < 1 || taps > MAX_TAPS || !conv_out || (taps > 1 && (!conv_state || !state_slot))))
    MI_REFUSE("branch_depth: %d convolution taps (1 to %d), with a state and an output", taps, MAX_TAPS);
  if (conv_w && taps > 1 && conv_stride < (long long)(taps - 1) * H) MI_REFUSE("branch_depth: the state's rows are too short");
  BranchDepthArgs a = {stream, branch, branch_stride, w, b, eps, stream_out, copy, first, results, n_prev, avg,
                       avg_out, conv_w, taps, conv_state, conv_stride, state_slot, conv_out, M, H};
  const size_t smem = branch ? (size_t)H * sizeof(float) : 0;
  if (smem > 200 * 1024) MI_REFUSE("branch_depth: a row of %d floats does not fit in shared memory", H);
  const bool vec = H % 4 == 0 && branch_stride % 4 == 0 && conv_stride % 4 == 0 && mi_aligned(stream, 16) &&
                   mi_aligned(branch, 16) && mi_aligned(w, 16) && mi_aligned(b, 16) && mi_aligned(stream_out, 16) &&
                   mi_aligned(copy, 16) && mi_aligned(first, 16) && mi_aligned(results, 16) && mi_aligned(avg_out, 16) &&
                   mi_aligned(conv_w, 16) && mi_aligned(conv_state, 16) && mi_aligned(conv_out, 16);
  const int per = vec ? H / 4 : H;
  if (vec && per <= ROW_MAX_THREADS) {      // (the choice depends on the width alone: a row's bits do not depend on the step)
    const int row_threads = (per + 31) / 32 * 32;
#define MI_ROW(T)                                                                                             \
  do {                                                                                                        \
    if (n_prev > 0 && conv_w) MI_LAUNCH((branch_depth_row_kernel<T, true, true>), M, row_threads, 0, cu_stream, a);   \
    else if (n_prev > 0) MI_LAUNCH((branch_depth_row_kernel<T, true, false>), M, row_threads, 0, cu_stream, a);       \
    else if (conv_w) MI_LAUNCH((branch_depth_row_kernel<T, false, true>), M, row_threads, 0, cu_stream, a);           \
    else MI_LAUNCH((branch_depth_row_kernel<T, false, false>), M, row_threads, 0, cu_stream, a);                      \
  } while (0)
    if (dtype == MI_DTYPE_F32) MI_ROW(float);
    else if (dtype == MI_DTYPE_BF16) MI_ROW(bf16);
    else MI_REFUSE("branch_depth: unknown dtype %d", dtype);
#undef MI_ROW
    MI_RETURN_LAUNCH_STATUS();
  }
  const int threads = per >= 1024 ? 512 : (per >= 256 ? 256 : 128);
#define MI_GO(T, V)                                                                                         \
  do {                                                                                                      \
    auto kern = branch_depth_kernel<T, V>;                                                                  \
    if (smem > 48 * 1024) {                                                                                 \
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
      if (e != cudaSuccess) return (int)e;                                                                  \
    }                                                                                                       \
    MI_LAUNCH(kern, M, threads, smem, cu_stream, a);                                                        \
  } while (0)
  if (dtype == MI_DTYPE_F32) {
    if (vec) MI_GO(float, 4); else MI_GO(float, 1);
  } else if (dtype == MI_DTYPE_BF16) {
    if (vec) MI_GO(bf16, 4); else MI_GO(bf16, 1);
  } else {
    MI_REFUSE("branch_depth: unknown dtype %d", dtype);
  }
#undef MI_GO
  MI_RETURN_LAUNCH_STATUS();
}

// One thread: V channels of a tile of CONV_TILE tokens of one request; with TAPS > 0 (that many taps) all of
// the tile's inputs are asked for before the first sum.  The threads of a request's first tile read the
// state and, behind that, replace it (nobody else touches it).
#define CONV_TILE 8
template <typename TX, typename T, int V, int TAPS>
__global__ void input_conv_kernel(const TX* __restrict__ x, int x_stride, const float* __restrict__ w, int taps,
                                  float* __restrict__ state, long long state_stride, const int* __restrict__ q_start,
                                  const int* __restrict__ q_len, const int* __restrict__ state_slot,
                                  T* __restrict__ out, int H) {
  mi_pdl_enter();
  const int k = V * (blockIdx.x * blockDim.x + threadIdx.x);
  const int req = blockIdx.z, len = q_len[req];
  if (k >= H) return;
  const int row0 = q_start[req], before = taps - 1;
  float* tail = before > 0 ? state + (size_t)state_slot[req] * state_stride + k : nullptr;
  const TX* xr = x + (size_t)row0 * x_stride + k;
  auto input = [&](int t, float (&f)[V]) {            // portion token t; before the portion: the state
    if (t >= 0) Pack<TX, V>::load(xr + (size_t)t * x_stride, f);
    else Pack<float, V>::load(tail + (size_t)(before + t) * H, f);
  };
  // the first block walks the first two tiles: nobody else's reach back into the state (at most 15 inputs)
  const int tile0 = blockIdx.y == 0 ? 0 : blockIdx.y + 1, tiles = blockIdx.y == 0 ? 2 : 1;
  for (int t0 = tile0 * CONV_TILE; t0 < min(len, (tile0 + tiles) * CONV_TILE); t0 += CONV_TILE) {
    if (TAPS > 0) {
      constexpr int N = TAPS > 0 ? TAPS : 1;
      float in[CONV_TILE + N - 1][V], wj[N][V];
#pragma unroll
      for (int i = 0; i < CONV_TILE + TAPS - 1; ++i)
        if (t0 + i - (TAPS - 1) < len) input(t0 + i - (TAPS - 1), in[i]);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) Pack<float, V>::load(w + (size_t)j * H + k, wj[j]);
#pragma unroll
      for (int t = 0; t < CONV_TILE; ++t) {
        if (t0 + t < len) {
          float acc[V];
#pragma unroll
          for (int i = 0; i < V; ++i) acc[i] = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j)
#pragma unroll
            for (int i = 0; i < V; ++i) acc[i] = fmaf(wj[j][i], in[t + j][i], acc[i]);
#pragma unroll
          for (int i = 0; i < V; ++i) acc[i] = in[t + TAPS - 1][i] + acc[i];
          Pack<T, V>::store(out + (size_t)(row0 + t0 + t) * H + k, acc);
        }
      }
    } else {
      const int t1 = min(len, t0 + CONV_TILE);
      for (int t = t0; t < t1; ++t) {
        float acc[V], wj[V], f[V];
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = 0.f;
        for (int j = 0; j < taps; ++j) {
          input(t - before + j, f);
          Pack<float, V>::load(w + (size_t)j * H + k, wj);
#pragma unroll
          for (int i = 0; i < V; ++i) acc[i] = fmaf(wj[i], f[i], acc[i]);
        }
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = f[i] + acc[i];          // f: the current token, read last
        Pack<T, V>::store(out + (size_t)(row0 + t) * H + k, acc);
      }
    }
  }
  if (blockIdx.y == 0)
    for (int j = 0; j < before; ++j) {                 // ascending: a slot is read before it is replaced
      float f[V];
      input(len - before + j, f);
      Pack<float, V>::store(tail + (size_t)j * H, f);
    }
}

// x_dtype: the input is fp32 (a residual stream) or in the compute dtype
extern "C" int mi_input_conv(const void* x, int x_stride, int x_dtype, const float* w, int taps, float* state,
                             long long state_stride, const int* q_start, const int* q_len, const int* state_slot,
                             void* out, int n_requests, int max_len, int H, int dtype, cudaStream_t stream) {
  if (n_requests <= 0 || max_len <= 0) return 0;
  if (H <= 0 || taps < 1 || taps > MAX_TAPS) MI_REFUSE("input_conv: width %d, %d taps (1 to %d)", H, taps, MAX_TAPS);
  if (taps > 1 && (!state || state_stride < (long long)(taps - 1) * H)) MI_REFUSE("input_conv: the state's rows are too short");
  if (n_requests > 65535) MI_REFUSE("input_conv: %d requests in one step", n_requests);
  const bool vec = H % 4 == 0 && x_stride % 4 == 0 && state_stride % 4 == 0 && mi_aligned(x, 16) && mi_aligned(w, 16) &&
                   mi_aligned(state, 16) && mi_aligned(out, 16);
  const int per = vec ? H / 4 : H;
  const int threads = 128;
  const long long tiles = (max_len + CONV_TILE - 1) / CONV_TILE;
  if (tiles > 65535) MI_REFUSE("input_conv: a portion of %d tokens", max_len);
  const dim3 grid((unsigned)((per + threads - 1) / threads), (unsigned)(tiles > 2 ? tiles - 1 : 1), (unsigned)n_requests);
#define MI_GO(TX, T, V, TAPS)                                                                                      \
  MI_LAUNCH((input_conv_kernel<TX, T, V, TAPS>), grid, threads, 0, stream, (const TX*)x, x_stride, w, taps, state, \
            state_stride, q_start, q_len, state_slot, (T*)out, H)
#define MI_PICK(TX, T)                          \
  do {                                          \
    if (vec && taps == 2) MI_GO(TX, T, 4, 2);   \
    else if (vec && taps == 3) MI_GO(TX, T, 4, 3); \
    else if (vec && taps == 4) MI_GO(TX, T, 4, 4); \
    else if (vec) MI_GO(TX, T, 4, 0);           \
    else MI_GO(TX, T, 1, 0);                    \
  } while (0)
  if (dtype == MI_DTYPE_F32 && x_dtype == MI_DTYPE_F32) MI_PICK(float, float);
  else if (dtype == MI_DTYPE_BF16 && x_dtype == MI_DTYPE_F32) MI_PICK(float, bf16);
  else if (dtype == MI_DTYPE_BF16 && x_dtype == MI_DTYPE_BF16) MI_PICK(bf16, bf16);
  else MI_REFUSE("input_conv: unsupported dtypes %d (input) and %d", x_dtype, dtype);
#undef MI_PICK
#undef MI_GO
  MI_RETURN_LAUNCH_STATUS();
}
