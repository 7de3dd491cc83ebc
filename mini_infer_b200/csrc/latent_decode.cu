// The small products around latent attention in steps of single tokens (bfloat16), each fused with what stands
// beside it.  Weights do not depend on the kernels before, so every thread asks for its first pieces of them
// before it waits for those.
//
//   mi_latent_query   qfull[t, h] = [W_h q_un(t, h), rotate(q_rot(t, h))]: a head's unrotated query mapped into
//                     the latent's space (W_h = uk_t[h], [rank, d]) and its rotated part, at the token's position.
//   mi_latent_value   out[t, h] = act(gate) * scale * W_h latent(t, h) with W_h = uv[h], [dv, rank]: the heads'
//                     values from the weighted sums of latents.  The sums come as attention_rows leaves them:
//                     runs of keys, unnormalised, with their maxima (log2) and denominators, which are merged
//                     here in a fixed order together with the head's sink; or as finished bfloat16 rows.
//
// fp32 arithmetic throughout; one rounding of every result.
#include "common.cuh"

MI_DEFINE_ERROR_API()

#define Q_ROWS 64          // rows of W per block: two neighbouring threads share a row
#define Q_MAX_TOKENS 16
#define Q_MAX_D 128
#define Q_MAX_PIECES (Q_MAX_D / 16)   // 16-byte pieces of half a row
#define Q_MAX_ROT 512

__device__ __forceinline__ void unpack8(const uint4& v, float (&f)[8]) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 p = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[i]));
    f[2 * i] = p.x;
    f[2 * i + 1] = p.y;
  }
}

// grid = (heads, blocks of Q_ROWS rows of W, then one more for the rotation)
__global__ void __launch_bounds__(128)
latent_query_kernel(const bf16* __restrict__ q, int q_stride, const bf16* __restrict__ uk_t, int M, int n, int d, int rank,
                    int rd, int rot, int interleaved, const int* __restrict__ positions,
                    const double* __restrict__ freq, bf16* __restrict__ qfull) {
  mi_pdl_launch_dependents();
  __shared__ __align__(16) float qs[Q_MAX_TOKENS][Q_MAX_D];
  const int h = blockIdx.x, tid = threadIdx.x, dk = rank + rd, qh = d + rd;
  if (blockIdx.y == gridDim.y - 1) {
    mi_pdl_wait();
    const int half = rot >> 1, work = half + (rd - rot);       // pairs, then the dimensions that pass
    for (int idx = tid; idx < M * work; idx += blockDim.x) {
      const int t = idx / work, i = idx - t * work;
      const bf16* src = q + (size_t)t * q_stride + (size_t)h * qh + d;
      bf16* dst = qfull + ((size_t)t * n + h) * dk + rank;
      if (i >= half) {
        dst[rot + i - half] = src[rot + i - half];
        continue;
      }
      double a = (double)positions[t] * freq[i];
      a -= 6.283185307179586476925 * rint(a * 0.15915494309189533577);
      float s, c, y1, y2;
      sincosf((float)a, &s, &c);
      const int k1 = interleaved ? 2 * i : i, k2 = interleaved ? 2 * i + 1 : i + half;
      mi_rotate(mi_to_float(src[k1]), mi_to_float(src[k2]), s, c, y1, y2);
      dst[k1] = mi_from_float<bf16>(y1);
      dst[k2] = mi_from_float<bf16>(y2);
    }
    return;
  }
  const int row = blockIdx.y * Q_ROWS + (tid >> 1), part = tid & 1;
  const int pieces = d >> 3, mine = (pieces - part + 1) >> 1;          // pieces part, part + 2, ...
  uint4 w[Q_MAX_PIECES];
#pragma unroll
  for (int i = 0; i < Q_MAX_PIECES; ++i) {
    w[i] = make_uint4(0u, 0u, 0u, 0u);
    if (i < mine && row < rank)
      w[i] = *reinterpret_cast<const uint4*>(uk_t + ((size_t)h * rank + row) * d + (2 * i + part) * 8);
  }
  mi_pdl_wait();
  for (int idx = tid; idx < M * pieces; idx += blockDim.x) {
    const int t = idx / pieces, c = idx - t * pieces;
    float f[8];
    unpack8(*reinterpret_cast<const uint4*>(q + (size_t)t * q_stride + (size_t)h * qh + c * 8), f);
#pragma unroll
    for (int j = 0; j < 8; ++j) qs[t][c * 8 + j] = f[j];
  }
  __syncthreads();
  float wf[Q_MAX_PIECES][8];
#pragma unroll
  for (int i = 0; i < Q_MAX_PIECES; ++i) unpack8(w[i], wf[i]);
  for (int t = 0; t < M; ++t) {
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < Q_MAX_PIECES; ++i) {
      if (i < mine) {
        const float4 x0 = *reinterpret_cast<const float4*>(&qs[t][(2 * i + part) * 8]);
        const float4 x1 = *reinterpret_cast<const float4*>(&qs[t][(2 * i + part) * 8 + 4]);
        acc = fmaf(wf[i][0], x0.x, acc); acc = fmaf(wf[i][1], x0.y, acc);
        acc = fmaf(wf[i][2], x0.z, acc); acc = fmaf(wf[i][3], x0.w, acc);
        acc = fmaf(wf[i][4], x1.x, acc); acc = fmaf(wf[i][5], x1.y, acc);
        acc = fmaf(wf[i][6], x1.z, acc); acc = fmaf(wf[i][7], x1.w, acc);
      }
    }
    acc += __shfl_xor_sync(0xffffffffu, acc, 1);
    if (part == 0 && row < rank) qfull[((size_t)t * n + h) * dk + row] = mi_from_float<bf16>(acc);
  }
}

extern "C" int mi_latent_query(const void* q, int q_stride, const void* uk_t, int M, int n, int d, int rank, int rd,
                               int rot, int interleaved, const int* positions, const double* freq, void* qfull,
                               cudaStream_t stream) {
  if (M <= 0) return 0;
  if (M > Q_MAX_TOKENS) MI_REFUSE("latent_query: %d tokens (up to %d)", M, Q_MAX_TOKENS);
  if (n <= 0 || d < 8 || d > Q_MAX_D || d % 8 || rank <= 0 || rd < 0 || (d + rd) % 8 || q_stride % 8)
    MI_REFUSE("latent_query: %d heads of %d + %d, latents of %d, rows of %d are not taken", n, d, rd, rank, q_stride);
  if (rot < 0 || rot > rd || (rot & 1) || rot > Q_MAX_ROT || (rot > 0 && (!positions || !freq)))
    MI_REFUSE("latent_query: %d rotated dimensions of %d need positions and frequencies", rot, rd);
  if (!mi_aligned(q, 16) || !mi_aligned(uk_t, 16)) MI_REFUSE("latent_query: operands must be 16-byte aligned");
  const dim3 grid((unsigned)n, (unsigned)((rank + Q_ROWS - 1) / Q_ROWS + 1));
  MI_LAUNCH((latent_query_kernel), grid, 128, 0, stream, (const bf16*)q, q_stride, (const bf16*)uk_t, M, n, d, rank, rd, rot,
            interleaved, positions, freq, (bf16*)qfull);
  MI_RETURN_LAUNCH_STATUS();
}

#define V_THREADS 512
#define V_RUNS 16           // runs of keys whose sums are asked for before their weights are known
#define V_PIECES 8          // 16-byte pieces of W in flight per thread: with eight threads a row, latents of 512 in one go
#define V_MAX_SPLITS 64
#define RUN_ROWS 16         // rows of a tile of attention_rows in a step of single tokens

// grid = (heads, tokens).  Eight neighbouring threads share a row of W.
__global__ void __launch_bounds__(V_THREADS)
latent_value_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int n_splits,
                    const bf16* __restrict__ latent, const float* __restrict__ sinks, const bf16* __restrict__ uv, int n,
                    int rank, int dv, const bf16* __restrict__ gate, int gate_stride, int per_head, int act, float scale,
                    bf16* __restrict__ out, int out_stride) {
  mi_pdl_launch_dependents();
  extern __shared__ __align__(16) float lat[];       // [rank]
  __shared__ float weight[V_MAX_SPLITS];
  __shared__ float inv_l;
  constexpr float LOG2E = 1.4426950408889634f;
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane8 = tid & 7;
  const int pieces = rank >> 3;
  const bf16* wh = uv + (size_t)h * dv * rank;
  uint4 w[V_PIECES];
  auto fetch = [&](int row, int c0) {
#pragma unroll
    for (int i = 0; i < V_PIECES; ++i) {
      const int c = c0 + i * 8 + lane8;
      w[i] = make_uint4(0u, 0u, 0u, 0u);
      if (row < dv && c < pieces) w[i] = *reinterpret_cast<const uint4*>(wh + (size_t)row * rank + c * 8);
    }
  };
  fetch(tid >> 3, 0);
  mi_pdl_wait();
  if (n_splits > 1) {
    const int head_tiles = (n + RUN_ROWS - 1) / RUN_ROWS;
    const size_t unit = (size_t)t * head_tiles + h / RUN_ROWS;
    const int r = h % RUN_ROWS;
    const float* pml = part_ml + (unit * n_splits * RUN_ROWS + r) * 2;
    const float* po = part_o + (unit * n_splits * RUN_ROWS + r) * rank;
    float v[V_RUNS];                 // this thread's column of the first runs
    auto ask = [&](int s0, int c) {
#pragma unroll
      for (int u = 0; u < V_RUNS; ++u)
        v[u] = (s0 + u < n_splits && c < rank) ? po[(size_t)(s0 + u) * RUN_ROWS * rank + c] : 0.f;
    };
    ask(0, tid);
    if (tid < 32) {                  // lane s: runs s and s + 32 (their maxima and denominators)
      float2 ml[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int s = tid + 32 * k;
        ml[k] = s < n_splits ? *reinterpret_cast<const float2*>(pml + (size_t)s * RUN_ROWS * 2) : make_float2(-INFINITY, 0.f);
      }
      const float sink2 = sinks ? sinks[h] * LOG2E : -INFINITY;
      const float mf = fmaxf(mi_warp_max(fmaxf(ml[0].x, ml[1].x)), sink2);
      float l = 0.f;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const float ws = ml[k].x == -INFINITY ? 0.f : exp2f(ml[k].x - mf);
        weight[tid + 32 * k] = ws;
        l += mi_warp_sum(ml[k].y * ws);
      }
      if (sinks) l += exp2f(sink2 - mf);
      if (tid == 0) inv_l = l > 0.f ? 1.f / l : 0.f;
    }
    __syncthreads();
    const float inv = inv_l;
    for (int c = tid; c < rank; c += V_THREADS) {
      float sum = 0.f;
      for (int s0 = 0; s0 < n_splits; s0 += V_RUNS) {     // added in order
        if (s0 || c != tid) ask(s0, c);
#pragma unroll
        for (int u = 0; u < V_RUNS; ++u) sum = fmaf(v[u], s0 + u < V_MAX_SPLITS ? weight[s0 + u] : 0.f, sum);
      }
      lat[c] = sum * inv;
    }
  } else {
    const bf16* src = latent + ((size_t)t * n + h) * rank;
    for (int c = tid; c < rank; c += V_THREADS) lat[c] = mi_to_float(src[c]);
  }
  __syncthreads();
  for (int row0 = 0; row0 < dv; row0 += V_THREADS / 8) {
    const int row = row0 + (tid >> 3);
    float acc = 0.f;
    for (int c0 = 0; c0 < pieces; c0 += 8 * V_PIECES) {
      if (row0 || c0) fetch(row, c0);
#pragma unroll
      for (int i = 0; i < V_PIECES; ++i) {
        const int c = c0 + i * 8 + lane8;
        if (c < pieces) {
          float f[8];
          unpack8(w[i], f);
          const float4 x0 = *reinterpret_cast<const float4*>(lat + c * 8), x1 = *reinterpret_cast<const float4*>(lat + c * 8 + 4);
          acc = fmaf(f[0], x0.x, acc); acc = fmaf(f[1], x0.y, acc); acc = fmaf(f[2], x0.z, acc); acc = fmaf(f[3], x0.w, acc);
          acc = fmaf(f[4], x1.x, acc); acc = fmaf(f[5], x1.y, acc); acc = fmaf(f[6], x1.z, acc); acc = fmaf(f[7], x1.w, acc);
        }
      }
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if (lane8 == 0 && row < dv) {
      acc *= scale;
      if (gate) {
        const float g = mi_to_float(gate[(size_t)t * gate_stride + (per_head ? h : h * dv + row)]);
        const float sg = 1.f / (1.f + expf(-g));
        acc *= act == 2 ? g * sg : sg;
      }
      out[(size_t)t * out_stride + h * dv + row] = mi_from_float<bf16>(acc);
    }
  }
}

// part_o / part_ml / n_splits: what mi_attention_rows left with merge = 0 (tiles of 16 rows, one token per request);
// n_splits 1: `latent` [M, n * rank] instead.  act: 1 sigmoid, 2 SiLU of `gate` ([M, n] with per_head, else [M, n * dv]).
extern "C" int mi_latent_value(const float* part_o, const float* part_ml, int n_splits, const void* latent,
                               const float* sinks, const void* uv, int M, int n, int rank, int dv, const void* gate,
                               int gate_stride, int per_head, int act, float scale, void* out, int out_stride,
                               cudaStream_t stream) {
  if (M <= 0) return 0;
  if (M > 65535 || n <= 0 || rank <= 0 || rank % 8 || dv <= 0) MI_REFUSE("latent_value: %d heads, latents of %d, values of %d are not taken", n, rank, dv);
  if (n_splits < 1 || n_splits > V_MAX_SPLITS || (n_splits > 1 ? !part_o || !part_ml : !latent))
    MI_REFUSE("latent_value: 1 to %d runs of keys with their sums, or finished rows", V_MAX_SPLITS);
  if (gate && act != 1 && act != 2) MI_REFUSE("latent_value: unknown gate %d", act);
  if (!mi_aligned(uv, 16) || !mi_aligned(part_ml, 8)) MI_REFUSE("latent_value: operands must be aligned");
  const size_t smem = (size_t)rank * sizeof(float);
  if (smem > 46 * 1024) MI_REFUSE("latent_value: a latent of %d does not fit in shared memory", rank);
  const dim3 grid((unsigned)n, (unsigned)M);
  MI_LAUNCH((latent_value_kernel), grid, V_THREADS, smem, stream, part_o, part_ml, n_splits, (const bf16*)latent, sinks,
            (const bf16*)uv, n, rank, dv, (const bf16*)gate, gate_stride, per_head, act, scale, (bf16*)out, out_stride);
  MI_RETURN_LAUNCH_STATUS();
}
