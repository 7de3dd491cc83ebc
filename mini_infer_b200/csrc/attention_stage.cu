// What stands around a paged attention: the preparation of its queries, keys and values behind the projection, and
// what is done to its heads before the output projection.
//
//   mi_rope_angles       per token the sines, then the cosines of position * freq[i], both times `mult`; the angle
//                        is formed and reduced to [-pi, pi] in double precision.
//   mi_conv_rope_store   queries, keys and values (columns [q | k | v] of one packed projection) pass a causal
//                        convolution per channel over `taps` tokens; queries and keys are then rotated in the half
//                        layout on their first `rot` dimensions (i pairs with i + rot/2); queries go to a tensor of
//                        their own, keys and values to their cache pages.  The projection stays as it is: a later
//                        tile of the portion reads it for its first tokens.  Before a portion's first token stand
//                        the request's last taps - 1 projected rows (fp32 state, oldest first), which the block of
//                        the portion's first tile moves on when it has read them.
//   mi_split_maps_store  queries and keys that come as two maps per head side by side: a key's row in the cache is
//                        [map 1 | map 2 | zeros], a query of map 1 becomes a row with map 1 in its place and zeros
//                        elsewhere, one of map 2 likewise, so that an ordinary attention over 2 nq query heads
//                        scores each map by itself.  Queries are multiplied by 1 + coef ln(floor((p + 1) / every) + 1).
//   mi_combine_maps      per token and head, from the two maps' outputs a1, a2 (heads 2h and 2h + 1):
//                        o = a1 - lam a2, times mult / sqrt(mean(o^2) + eps), times sigmoid(gate[t, h]) (optional).
//
// Every value is rounded once; everything before that is fp32.
#include "common.cuh"

MI_DEFINE_ERROR_API()

#define STAGE_TILE 16      // tokens per tile of mi_conv_rope_store
#define STAGE_THREADS 128
#define STAGE_RUN 4        // consecutive tokens that a thread of mi_conv_rope_store takes at a time
#define STAGE_MAX_TAPS 16  // taps - 1 rows of state: only a portion's first tile reads them

__global__ void rope_angles_kernel(const int* __restrict__ positions, const double* __restrict__ freq, float mult,
                                   float* __restrict__ out, int M, int half) {
  mi_pdl_enter();
  const int idx = blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= M * half) return;
  const int t = idx / half, i = idx - t * half;
  double a = (double)positions[t] * freq[i];
  a -= 6.283185307179586476925 * rint(a * 0.15915494309189533577);
  float s, c;
  sincosf((float)a, &s, &c);
  out[(size_t)t * 2 * half + i] = s * mult;
  out[(size_t)t * 2 * half + half + i] = c * mult;
}

extern "C" int mi_rope_angles(const int* positions, const double* freq, float mult, float* out, int M, int half,
                              cudaStream_t stream) {
  if (M <= 0 || half <= 0) return 0;
  if ((long long)M * half > 0x7fffffffLL) MI_REFUSE("rope_angles: too many angles for one launch");
  MI_LAUNCH(rope_angles_kernel, (unsigned)((M * half + 127) / 128), 128, 0, stream, positions, freq, mult, out, M, half);
  MI_RETURN_LAUNCH_STATUS();
}

// V consecutive values as one access (8 of bfloat16, or 4) or one by one (1).
template <typename T, int V>
struct Piece {
  float f[V];
  __device__ __forceinline__ void load(const T* p) {
    if constexpr (V == 8) {
      static_assert(V != 8 || sizeof(T) == 2, "eight values of bfloat16 are one access");
      const uint4 v = *reinterpret_cast<const uint4*>(p);
      const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[j]));
        f[2 * j] = g.x;
        f[2 * j + 1] = g.y;
      }
    } else if constexpr (V == 4) {
      Vec4<T> v;
      v.load(p);
      v.get(f);
    } else {
      f[0] = mi_to_float(p[0]);
    }
  }
  __device__ __forceinline__ void store(T* p) const {
    if constexpr (V == 8) {
      uint32_t w[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const __nv_bfloat162 g = __floats2bfloat162_rn(f[2 * j], f[2 * j + 1]);
        w[j] = *reinterpret_cast<const uint32_t*>(&g);
      }
      *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
    } else if constexpr (V == 4) {
      Vec4<T> v;
      v.set(f);
      v.store(p);
    } else {
      p[0] = mi_from_float<T>(f[0]);
    }
  }
};

// A block takes one head and one tile of tokens; a thread convolves V channels of it for runs of STAGE_RUN tokens.
// Dimensions that pass go straight to their destination, those that are turned through shared memory (`turned`,
// [STAGE_TILE][rot] fp32), where the turn finds its partner.  TAPS > 0: that many taps; weights and inputs of a run are
// in registers, all inputs asked for before the first is used.  0: `taps` of them, read as they are used.
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(STAGE_THREADS)
conv_rope_store_kernel(const T* __restrict__ packed, int stride, const float* __restrict__ weight, int taps_any,
                       float* __restrict__ state, long long state_stride, const int* __restrict__ state_slot,
                       const int* __restrict__ q_start, const int* __restrict__ q_len, const int* __restrict__ tile_req,
                       const int* __restrict__ tile_tok0, int nq, int nkv, int d, int dv, int rot,
                       const float* __restrict__ angles, const int* __restrict__ slots, T* __restrict__ q_out,
                       T* __restrict__ kcache, T* __restrict__ vcache, int page_size) {
  mi_pdl_enter();
  constexpr int EPC = 16 / (int)sizeof(T);
  constexpr int NW = TAPS > 0 ? TAPS : 1, NH = TAPS > 1 ? TAPS - 1 : 1;
  constexpr int NI = TAPS > 0 ? STAGE_RUN + TAPS - 1 : 1;      // inputs of a run
  extern __shared__ __align__(16) float turned[];
  __shared__ long long to[STAGE_TILE];                         // where a token's row begins at its destination
  __shared__ int swz[STAGE_TILE];                              // and the permutation of its 16-byte pieces
  const int taps = TAPS > 0 ? TAPS : taps_any, C = (nq + nkv) * d + nkv * dv;
  const int tile = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
  const int b = tile_req[tile], tok0 = tile_tok0[tile];
  const int ql = q_len[b], qs = q_start[b];
  const int ntok = min(STAGE_TILE, ql - tok0);
  const bool is_q = head < nq, is_v = head >= nq + nkv;
  const int width = is_v ? dv : d, turn = is_v ? 0 : rot, half = turn >> 1;
  const int base = is_v ? (nq + nkv) * d + (head - nq - nkv) * dv : head * d;      // the head's first channel
  float* past = state ? state + (long long)state_slot[b] * state_stride : nullptr;
  T* dst = is_q ? q_out : (is_v ? vcache : kcache);
  if (tid < ntok) {
    const int row = qs + tok0 + tid;
    if (is_q) {
      to[tid] = ((long long)row * nq + head) * d;
      swz[tid] = 0;
    } else {
      const int kvh = is_v ? head - nq - nkv : head - nq, slot = slots[row], page = slot / page_size;
      const int offset = slot - page * page_size;
      to[tid] = ((long long)(page * nkv + kvh) * page_size + offset) * width;
      swz[tid] = offset & mi_swizzle_mask_rows(width, (int)sizeof(T));
    }
  }
  auto put = [&](int tt, int k, const Piece<T, V>& p) {         // V values from dimension k on of the tile's token tt
    const int s = swz[tt];
    p.store(dst + to[tt] + (s ? (((k / EPC) ^ s) * EPC + k % EPC) : k));
  };
  // the projected values of V channels from c on at the portion's token src (negative: before the portion)
  auto input = [&](int src, int c, Piece<T, V>& u) {
    if (src >= 0) {
      u.load(packed + (size_t)(qs + src) * stride + c);
    } else {
      const float* p = past + (size_t)(taps - 1 + src) * C + c;
#pragma unroll
      for (int e = 0; e < V; ++e) u.f[e] = p[e];
    }
  };

  const int n_items = width / V, lanes = min(n_items, STAGE_THREADS), groups = STAGE_THREADS / lanes;
  const int group = tid / lanes, lane = tid - group * lanes;
  // every thread takes part in every round: the first one waits for `to` and `swz` between its loads and its stores
  bool first = true;
  for (int item = lane; item - lane < n_items; item += lanes) {
    const bool mine = item < n_items && group < groups;
    const int k = item * V, c = base + k;
    float w[NW][V];
    if (TAPS > 0 && mine) {
#pragma unroll
      for (int j = 0; j < NW; ++j) {
        Piece<float, V> p;
        p.load(weight + (size_t)j * C + c);
#pragma unroll
        for (int e = 0; e < V; ++e) w[j][e] = p.f[e];
      }
    }
    for (int run0 = 0; run0 < ntok; run0 += groups * STAGE_RUN) {
      const int run = run0 + group * STAGE_RUN, t0 = tok0 + run, n = mine ? min(STAGE_RUN, ntok - run) : 0;
      Piece<T, V> u[NI];
      if (TAPS > 0 && n > 0) {
        if (t0 >= TAPS - 1 && n == STAGE_RUN) {      // the usual run: no branch between the loads
          const T* p = packed + (size_t)(qs + t0 - (TAPS - 1)) * stride + c;
#pragma unroll
          for (int j = 0; j < NI; ++j) u[j].load(p + (size_t)j * stride);
        } else {
#pragma unroll
          for (int j = 0; j < NI; ++j)
            if (j < n + TAPS - 1) input(t0 - (TAPS - 1) + j, c, u[j]);
          if (TAPS > 1 && ql <= STAGE_RUN) {           // the portion is this run: its last inputs are the new state
#pragma unroll
            for (int r = 0; r < TAPS - 1; ++r)
#pragma unroll
              for (int e = 0; e < V; ++e) {
                float v = u[1 + r].f[e];
#pragma unroll
                for (int m = 2; m <= STAGE_RUN; ++m) v = n == m && m + r < NI ? u[m + r < NI ? m + r : 0].f[e] : v;
                past[(size_t)r * C + c + e] = v;
              }
          }
        }
      }
      if (first) {
        __syncthreads();
        first = false;
      }
#pragma unroll
      for (int i = 0; i < STAGE_RUN; ++i) {
        if (i < n) {
          Piece<T, V> y;
#pragma unroll
          for (int e = 0; e < V; ++e) y.f[e] = 0.f;
          if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j)
#pragma unroll
              for (int e = 0; e < V; ++e) y.f[e] = fmaf(w[j][e], u[i + j].f[e], y.f[e]);
          } else {
            for (int j = 0; j < taps; ++j) {
              Piece<T, V> v;
              input(t0 + i - taps + 1 + j, c, v);
#pragma unroll
              for (int e = 0; e < V; ++e) y.f[e] = fmaf(weight[(size_t)j * C + c + e], v.f[e], y.f[e]);
            }
          }
          if (k < turn) {
            Piece<float, V> p;
#pragma unroll
            for (int e = 0; e < V; ++e) p.f[e] = y.f[e];
            p.store(turned + (run + i) * turn + k);
          } else {
            put(run + i, k, y);
          }
        }
      }
    }
  }
  __syncthreads();      // the turned dimensions are in shared memory; this block, the only reader of its state, has read it
  if (turn) {
    const int pieces = turn / V;
    for (int idx = tid; idx < ntok * pieces; idx += STAGE_THREADS) {
      const int tt = idx / pieces, k = (idx - tt * pieces) * V, i = k < half ? k : k - half;
      const float* sn = angles + (size_t)(qs + tok0 + tt) * turn + i;
      Piece<float, V> x, z, s, o;
      x.load(turned + tt * turn + i);
      z.load(turned + tt * turn + half + i);
      s.load(sn);
      o.load(sn + half);
      Piece<T, V> y;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float y1, y2;
        mi_rotate(x.f[e], z.f[e], s.f[e], o.f[e], y1, y2);
        y.f[e] = k < half ? y1 : y2;
      }
      put(tt, k, y);
    }
  }
  if (tok0 == 0 && past && !(TAPS > 0 && ql <= STAGE_RUN)) {
    auto moved = [&](int r, int k) {      // what row r of the state becomes: a later row, or one of the portion's last
      const int src = ql - (taps - 1) + r;
      return src >= 0 ? mi_to_float(packed[(size_t)(qs + src) * stride + base + k]) : past[(size_t)(r + ql) * C + base + k];
    };
    for (int k = tid; k < width; k += STAGE_THREADS) {
      if constexpr (TAPS > 0) {               // all rows are asked for before the first is written
        float v[NH];
#pragma unroll
        for (int r = 0; r < TAPS - 1; ++r) v[r] = moved(r, k);
#pragma unroll
        for (int r = 0; r < TAPS - 1; ++r) past[(size_t)r * C + base + k] = v[r];
      } else {
        for (int r = 0; r < taps - 1; ++r)    // ascending: a row that moves up is read before it is written over
          past[(size_t)r * C + base + k] = moved(r, k);
      }
    }
  }
}

extern "C" int mi_conv_rope_store_tile_tokens() { return STAGE_TILE; }

extern "C" int mi_conv_rope_store(const void* packed, int stride, const float* weight, int taps, float* state,
                                  long long state_stride, const int* state_slot, const int* q_start, const int* q_len,
                                  const int* tile_req, const int* tile_tok0, int n_tiles, int nq, int nkv, int d, int dv,
                                  int rot, const float* angles, const int* slots, void* q_out, void* kcache,
                                  void* vcache, int page_size, int dtype, cudaStream_t stream) {
  if (n_tiles <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || d <= 0 || dv <= 0) MI_REFUSE("conv_rope_store: bad sizes");
  const int C = (nq + nkv) * d + nkv * dv;
  if (stride < C) MI_REFUSE("conv_rope_store: rows of %d values hold no %d channels", stride, C);
  if (taps < 1 || taps > STAGE_MAX_TAPS) MI_REFUSE("conv_rope_store: 1 to %d taps, not %d", STAGE_MAX_TAPS, taps);
  if (taps > 1 && (!state || !state_slot || state_stride < (long long)(taps - 1) * C))
    MI_REFUSE("conv_rope_store: %d taps need a state of %d rows", taps, taps - 1);
  if (rot < 0 || rot % 2 || rot > d || (rot && !angles)) MI_REFUSE("conv_rope_store: bad rotation of %d of %d dimensions", rot, d);
  if (!slots || !kcache || !vcache || page_size <= 0) MI_REFUSE("conv_rope_store: keys and values need slots and pages");
  const int n_heads = nq + 2 * nkv;
  if (n_heads > 65535) MI_REFUSE("conv_rope_store: too many heads for one launch");
  const size_t piece = dtype == MI_DTYPE_F32 ? 16 : 8;
  const bool four = d % 4 == 0 && dv % 4 == 0 && rot % 8 == 0 && stride % 4 == 0 && mi_aligned(packed, piece) &&
                    mi_aligned(q_out, piece) && mi_aligned(kcache, 16) && mi_aligned(vcache, 16) && mi_aligned(weight, 16) &&
                    mi_aligned(angles, 16);
  const size_t smem = (size_t)STAGE_TILE * rot * sizeof(float);
  if (smem > 47 * 1024) MI_REFUSE("conv_rope_store: %d rotated dimensions do not fit in shared memory", rot);
  const dim3 grid((unsigned)n_tiles, (unsigned)n_heads);
#define MI_CONV(T, V, TAPS)                                                                                           \
  MI_LAUNCH((conv_rope_store_kernel<T, V, TAPS>), grid, STAGE_THREADS, smem, stream, (const T*)packed, stride, weight,   \
            taps, taps > 1 ? state : (float*)nullptr, state_stride, state_slot, q_start, q_len, tile_req, tile_tok0,  \
            nq, nkv, d, dv, rot, angles, slots, (T*)q_out, (T*)kcache, (T*)vcache, page_size)
#define MI_CONV_TAPS(T, V)                                                                                            \
  do {                                                                                                                \
    if (taps == 1) MI_CONV(T, V, 1);                                                                                  \
    else if (taps == 2) MI_CONV(T, V, 2);                                                                                  \
    else if (taps == 3) MI_CONV(T, V, 3);                                                                             \
    else if (taps == 4) MI_CONV(T, V, 4);                                                                             \
    else MI_CONV(T, V, 0);                                                                                            \
  } while (0)
  if (dtype == MI_DTYPE_F32) {
    if (four) MI_CONV_TAPS(float, 4);
    else MI_CONV_TAPS(float, 1);
  } else if (dtype == MI_DTYPE_BF16) {
    if (four) MI_CONV_TAPS(bf16, 4);
    else MI_CONV_TAPS(bf16, 1);
  } else {
    MI_REFUSE("conv_rope_store: unknown dtype %d", dtype);
  }
#undef MI_CONV_TAPS
#undef MI_CONV
  MI_RETURN_LAUNCH_STATUS();
}

// grid = (tokens, parts): the pieces of a token's queries, key rows and values are numbered in one row
#define SPLIT_THREADS 128
template <typename T, int V>
__global__ void __launch_bounds__(SPLIT_THREADS)
split_maps_store_kernel(const T* __restrict__ packed, int stride, int k_off, int v_off, int nq, int nkv, int d, int rowd,
                        int dv, const int* __restrict__ positions, float coef, int every, const int* __restrict__ slots,
                        T* __restrict__ q_out, T* __restrict__ kcache, T* __restrict__ vcache, int page_size) {
  mi_pdl_enter();
  constexpr int EPC = 16 / (int)sizeof(T);
  const int t = blockIdx.x;
  const T* src = packed + (size_t)t * stride;
  const int slot = slots[t], page = slot / page_size, offset = slot - page * page_size;
  const int mk = mi_swizzle_mask_rows(rowd, (int)sizeof(T)), mv = mi_swizzle_mask_rows(dv, (int)sizeof(T));
  const float temp = coef != 0.f ? 1.f + coef * logf((float)((positions[t] + 1) / every + 1)) : 1.f;
  const int pr = rowd / V, pv = dv / V, n_q = 2 * nq * pr, n_k = nkv * pr, n_all = n_q + n_k + nkv * pv;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < n_all; i += gridDim.y * blockDim.x) {
    Piece<T, V> p;
#pragma unroll
    for (int e = 0; e < V; ++e) p.f[e] = 0.f;
    if (i < n_q) {
      const int h = i / pr, k = (i - h * pr) * V, own = k - (h & 1) * d;      // own: the column within the map
      if (own >= 0 && own < d) p.load(src + h * d + own);
#pragma unroll
      for (int e = 0; e < V; ++e) p.f[e] *= temp;
      p.store(q_out + ((size_t)t * 2 * nq + h) * rowd + k);
    } else if (i < n_q + n_k) {
      const int h = (i - n_q) / pr, k = (i - n_q - h * pr) * V;
      if (k < 2 * d) p.load(src + k_off + h * 2 * d + k);
      p.store(kcache + ((size_t)(page * nkv + h) * page_size + offset) * rowd + mi_swizzled(k, offset, mk, EPC));
    } else {
      const int h = (i - n_q - n_k) / pv, k = (i - n_q - n_k - h * pv) * V;
      p.load(src + v_off + h * dv + k);
      p.store(vcache + ((size_t)(page * nkv + h) * page_size + offset) * dv + mi_swizzled(k, offset, mv, EPC));
    }
  }
}

extern "C" int mi_split_maps_store(const void* packed, int stride, int k_off, int v_off, int M, int nq, int nkv, int d,
                                   int rowd, int dv, const int* positions, float coef, int every, const int* slots,
                                   void* q_out, void* kcache, void* vcache, int page_size, int dtype,
                                   cudaStream_t stream) {
  if (M <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || d <= 0 || dv <= 0 || rowd < 2 * d) MI_REFUSE("split_maps_store: bad sizes");
  if (every <= 0) MI_REFUSE("split_maps_store: the temperature grows every %d positions", every);
  if (!slots || !kcache || !vcache || page_size <= 0 || (coef != 0.f && !positions))
    MI_REFUSE("split_maps_store: keys and values need slots and pages, a temperature positions");
  const size_t piece = dtype == MI_DTYPE_F32 ? 16 : 8;
  auto fits = [&](int v, size_t align) {
    return d % v == 0 && rowd % v == 0 && dv % v == 0 && k_off % v == 0 && v_off % v == 0 && stride % v == 0 &&
           mi_aligned(packed, align) && mi_aligned(q_out, align) && mi_aligned(kcache, 16) && mi_aligned(vcache, 16);
  };
  const int V = dtype == MI_DTYPE_BF16 && fits(8, 16) ? 8 : (fits(4, piece) ? 4 : 1);
  const int items = (2 * nq + nkv) * rowd + nkv * dv, per = V * SPLIT_THREADS;
  int parts = (items + per - 1) / per;                 // a pass each for few tokens, two passes a block for many
  if (M >= 256) parts = (parts + 1) / 2;
  if (parts > 64) parts = 64;
  const dim3 grid((unsigned)M, (unsigned)parts);
#define MI_SPLIT(T, V)                                                                                               \
  MI_LAUNCH((split_maps_store_kernel<T, V>), grid, SPLIT_THREADS, 0, stream, (const T*)packed, stride, k_off, v_off, \
            nq, nkv, d, rowd, dv, positions, coef, every, slots, (T*)q_out, (T*)kcache, (T*)vcache, page_size)
  if (dtype == MI_DTYPE_F32) {
    if (V == 4) MI_SPLIT(float, 4);
    else MI_SPLIT(float, 1);
  } else if (dtype == MI_DTYPE_BF16) {
    if (V == 8) MI_SPLIT(bf16, 8);
    else if (V == 4) MI_SPLIT(bf16, 4);
    else MI_SPLIT(bf16, 1);
  } else {
    MI_REFUSE("split_maps_store: unknown dtype %d", dtype);
  }
#undef MI_SPLIT
  MI_RETURN_LAUNCH_STATUS();
}

// LANES lanes per (token, head), HELD pieces of V values per lane
#define COMBINE_THREADS 128
template <typename T, int V, int HELD, int LANES>
__global__ void __launch_bounds__(COMBINE_THREADS)
combine_maps_kernel(const T* __restrict__ heads, const T* __restrict__ gate, int gate_stride, T* __restrict__ out,
                    int out_stride, int M, int nq, int dv, float lam, float eps, float mult) {
  mi_pdl_enter();
  const int unit = blockIdx.x * (COMBINE_THREADS / LANES) + threadIdx.x / LANES, lane = threadIdx.x % LANES;
  const bool live = unit < M * nq;
  const int t = live ? unit / nq : 0, h = live ? unit - t * nq : 0;
  const T* a1 = heads + ((size_t)t * nq + h) * 2 * dv;
  const T* a2 = a1 + dv;
  const float g = gate ? mi_to_float(gate[(size_t)t * gate_stride + h]) : 0.f;
  Piece<T, V> o[HELD], b[HELD];
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int k = (lane + LANES * i) * V;
    if (k < dv) {
      o[i].load(a1 + k);
      b[i].load(a2 + k);
    }
  }
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < HELD; ++i)
    if ((lane + LANES * i) * V < dv) {
#pragma unroll
      for (int e = 0; e < V; ++e) {
        o[i].f[e] = fmaf(-lam, b[i].f[e], o[i].f[e]);
        sq += o[i].f[e] * o[i].f[e];
      }
    }
#pragma unroll
  for (int s = LANES / 2; s > 0; s >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, s);
  if (!live) return;
  float f = mult / sqrtf(sq / (float)dv + eps);
  if (gate) f *= 1.f / (1.f + expf(-g));
  T* dst = out + (size_t)t * out_stride + h * dv;
#pragma unroll
  for (int i = 0; i < HELD; ++i) {
    const int k = (lane + LANES * i) * V;
    if (k < dv) {
#pragma unroll
      for (int e = 0; e < V; ++e) o[i].f[e] *= f;
      o[i].store(dst + k);
    }
  }
}

extern "C" int mi_combine_maps(const void* heads, const void* gate, int gate_stride, void* out, int out_stride, int M,
                               int nq, int dv, float lam, float eps, float mult, int dtype, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (nq <= 0 || dv <= 0 || dv > 512) MI_REFUSE("combine_maps: bad sizes (%d heads, values of %d)", nq, dv);
  const size_t piece = dtype == MI_DTYPE_F32 ? 16 : 8;
  const bool four = dv % 4 == 0 && out_stride % 4 == 0 && mi_aligned(heads, piece) && mi_aligned(out, piece);
  const bool eight = dtype == MI_DTYPE_BF16 && dv % 8 == 0 && out_stride % 8 == 0 && mi_aligned(heads, 16) && mi_aligned(out, 16);
  const long long units = (long long)M * nq;
  if (units > 0x7fffffffLL - 64) MI_REFUSE("combine_maps: too many rows for one launch");
#define MI_COMBINE(T, V, HELD, LANES)                                                                                 \
  MI_LAUNCH((combine_maps_kernel<T, V, HELD, LANES>), (unsigned)((units * LANES + COMBINE_THREADS - 1) / COMBINE_THREADS), \
            COMBINE_THREADS, 0, stream, (const T*)heads, (const T*)gate, gate_stride, (T*)out, out_stride, M, nq, dv,   \
            lam, eps, mult)
#define MI_COMBINE_SIZE(T)                                                                                            \
  do {                                                                                                                \
    if (four && dv <= 128) MI_COMBINE(T, 4, 1, 32);                                                                   \
    else if (four) MI_COMBINE(T, 4, 4, 32);                                                                           \
    else MI_COMBINE(T, 1, 16, 32);                                                                                    \
  } while (0)
  if (dtype == MI_DTYPE_F32) MI_COMBINE_SIZE(float);
  else if (dtype == MI_DTYPE_BF16 && eight && dv <= 64) MI_COMBINE(bf16, 8, 1, 8);
  else if (dtype == MI_DTYPE_BF16 && eight && dv <= 128) MI_COMBINE(bf16, 8, 2, 8);
  else if (dtype == MI_DTYPE_BF16) MI_COMBINE_SIZE(bf16);
  else MI_REFUSE("combine_maps: unknown dtype %d", dtype);
#undef MI_COMBINE_SIZE
#undef MI_COMBINE
  MI_RETURN_LAUNCH_STATUS();
}
