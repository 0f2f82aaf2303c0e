// A mixture of experts around its matmuls, for weights kept as bf16 or fp32:
//   fb_route            router logits -> each token's k largest (by logit, or by softmax or sigmoid score), their weights, and where each
//                       choice's row goes (an identity expert's: nowhere): the touched experts' rows in whole tiles, a list of the tiles' experts, how many there are
//   fb_spread_rows      the tokens' rows to their choices' places
//   fb_grouped_matmul   rows of tiles by each tile's own matrix, any sizes, bf16 or fp32 (the tensor cores' form: fb_dense_grouped)
//
// Two layouts of the rows.  A few tokens: a tile a touched expert, holding all the tokens (nothing is gathered; an expert's
// weights, not its rows, are what such a step reads).  Many: each expert's choices one after another, filled up to whole tiles.
#include "launch.cuh"
#include "values.cuh"

namespace fb {

struct RouteArgs {
  const float* logits;  // [T, ld]
  int64_t T, ld;
  const float* bias;  // [n] or null
  int n, k, tile, shared;
  int real, scored;  // outputs 0 .. real - 1 are experts with rows; scored: 1 softmax, 2 sigmoid
  float scale;
  int as_scored;     // the weights are the scores, not over their sum
  int tiles;  // entries of tile_expert
  float* weights;       // [T, k]
  int32_t* ids;         // [T, k]
  int32_t* slots;       // [T, k]: the row of each choice
  int32_t* tile_expert; // [tiles, 3]: a tile's expert (n past those used), its expert's first tile and how many it has
  int32_t* live;        // [1] tiles used
  float* row_weights;   // each choice's weight at its row, or null
};

// a float as a number that orders like it (-0 as 0), above 0 for all of them
__device__ __forceinline__ uint32_t ordered(float v) {
  const uint32_t b = __float_as_uint(v + 0.f);
  return b & 0x80000000u ? ~b : b | 0x80000000u;
}
__device__ __forceinline__ float from_ordered(uint32_t b) { return __uint_as_float(b & 0x80000000u ? b & 0x7fffffffu : ~b); }

// the k largest of a token's logits or scores, the lower column first among equals, and their weights: a warp a token.  Up to 256
// outputs: the lanes hold the logits as ordered numbers, 0 once picked
__device__ __forceinline__ void route_token(const RouteArgs& a, int64_t t, int lane) {
  const float* z = a.logits + t * a.ld;
  float mine[2] = {-INFINITY, -INFINITY};  // lane j keeps the picks j and 32 + j
  int my_id[2] = {0, 0};
  float most = 0.f, norm = 1.f;  // scored by softmax: a score is exp(z - most) * norm
  if (a.scored == 1) {
    most = -INFINITY;
    for (int c = lane; c < a.n; c += 32) most = fmaxf(most, z[c]);
    most = warp_max(most);
    float sum = 0.f;
    for (int c = lane; c < a.n; c += 32) sum += expf(z[c] - most);
    norm = 1.f / warp_sum(sum);
  }
  auto score = [&](int c) { return a.scored == 1 ? expf(z[c] - most) * norm : sigmoid_f(z[c]); };
  // (sigmoids without a correction order as their logits do, which are never equal where those are not)
  auto chosen_by = [&](int c) { return (a.scored == 1 || (a.scored == 2 && a.bias) ? score(c) : z[c]) + (a.bias ? a.bias[c] : 0.f); };
  auto keep = [&](int j, float v, int at) {
    if (j < 32 && lane == j) mine[0] = v, my_id[0] = at;
    if (j >= 32 && lane == j - 32) mine[1] = v, my_id[1] = at;
  };
  if (a.n <= 256) {
    uint32_t held[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = 32 * i + lane;
      held[i] = c < a.n ? ordered(chosen_by(c)) : 0;
    }
    for (int j = 0; j < a.k; ++j) {
      uint32_t best = held[0];
      int at = lane;
#pragma unroll
      for (int i = 1; i < 8; ++i)
        if (held[i] > best) best = held[i], at = 32 * i + lane;
      const uint32_t top = __reduce_max_sync(0xffffffffu, best);
      at = __reduce_min_sync(0xffffffffu, best == top ? at : a.n);
      keep(j, from_ordered(top), at);
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (at == 32 * i + lane) held[i] = 0;
    }
  } else {
    float prev = INFINITY;
    int prev_at = -1;
    for (int j = 0; j < a.k; ++j) {
      float best = -INFINITY;
      int at = a.n;
      for (int c = lane; c < a.n; c += 32) {  // (what comes after the pick before in the order of the picks; columns rise: the first of equals stays)
        const float v = chosen_by(c);
        if ((v < prev || (v == prev && c > prev_at)) && (at == a.n || v > best)) best = v, at = c;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, at, o);
        if (oi < a.n && (at == a.n || ov > best || (ov == best && oi < at))) best = ov, at = oi;
      }
      if (at == a.n) at = 0;  // (only where a logit is not a number)
      prev = best, prev_at = at;
      keep(j, best, at);
    }
  }
  const float top = __shfl_sync(0xffffffffu, mine[0], 0);
  auto weight = [&](int i) { return lane + 32 * i >= a.k ? 0.f : a.scored ? score(min(my_id[i], a.n - 1)) : expf(mine[i] - top); };
  const float e0 = weight(0), e1 = weight(1), sum = a.as_scored ? 1.f : warp_sum(e0 + e1) + (a.scored ? 1e-20f : 0.f);
  if (lane < a.k) a.weights[t * a.k + lane] = e0 / sum * a.scale, a.ids[t * a.k + lane] = my_id[0];
  if (lane + 32 < a.k) a.weights[t * a.k + lane + 32] = e1 / sum * a.scale, a.ids[t * a.k + lane + 32] = my_id[1];
}

__global__ void __launch_bounds__(256) route_tokens_kernel(const RouteArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  const int64_t t = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (t < a.T) route_token(a, t, threadIdx.x & 31);
}

// one block: the choices' places.  `pick`: it makes the choices first
__global__ void __launch_bounds__(1024) route_places_kernel(const RouteArgs a, const int pick) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ int32_t route_smem[];  // [real] counts, then each expert's next row; [33] sums
  int32_t *count = route_smem, *sums = route_smem + a.real;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int e = tid; e < a.real; e += blockDim.x) count[e] = 0;
  if (pick)
    for (int64_t t = warp; t < a.T; t += 32) route_token(a, t, lane);
  __syncthreads();
  const int64_t choices = a.T * a.k;
  constexpr int BATCH = 8;  // a thread's choices on their way at once
  for (int64_t i0 = tid; i0 < choices; i0 += BATCH * 1024) {
    int e[BATCH];
#pragma unroll
    for (int b = 0; b < BATCH; ++b) e[b] = i0 + b * 1024 < choices ? a.ids[i0 + b * 1024] : -1;
#pragma unroll
    for (int b = 0; b < BATCH; ++b)
      if (e[b] >= 0 && e[b] < a.real) atomicAdd(count + e[b], 1);
  }
  __syncthreads();
  // tiles of each expert, scanned: a thread has a run of experts
  const int run = (a.real + 1023) / 1024, e0 = min(a.real, tid * run), e1 = min(a.real, e0 + run);
  auto tiles_of = [&](int e) { return a.shared ? (count[e] ? 1 : 0) : (count[e] + a.tile - 1) / a.tile; };
  int own = 0;
  for (int e = e0; e < e1; ++e) own += tiles_of(e);
  int before = own;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= o) before += v;
  }
  if (lane == 31) sums[warp] = before;
  __syncthreads();
  if (warp == 0) {
    int v = sums[lane];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += u;
    }
    sums[lane] = v;
  }
  __syncthreads();
  int first = before - own + (warp ? sums[warp - 1] : 0);
  const int used = sums[31];
  if (tid == 0) *a.live = used;
  for (int e = e0; e < e1; ++e) {
    const int n = tiles_of(e);
    for (int i = first; i < first + n && i < a.tiles; ++i) a.tile_expert[3 * i] = e, a.tile_expert[3 * i + 1] = first, a.tile_expert[3 * i + 2] = n;
    count[e] = first * a.tile;
    first += n;
  }
  for (int i = used + tid; i < a.tiles; i += blockDim.x) a.tile_expert[3 * i] = a.real, a.tile_expert[3 * i + 1] = a.tile_expert[3 * i + 2] = 0;
  __syncthreads();
  for (int64_t i0 = tid; i0 < choices; i0 += BATCH * 1024) {
    int e[BATCH];
#pragma unroll
    for (int b = 0; b < BATCH; ++b) e[b] = i0 + b * 1024 < choices ? a.ids[i0 + b * 1024] : -1;
#pragma unroll
    for (int b = 0; b < BATCH; ++b)
      if (e[b] >= 0) {
        const int64_t i = i0 + b * 1024;
        const int slot = e[b] >= a.real ? -1 : a.shared ? count[e[b]] + (int)(i / a.k) : atomicAdd(count + e[b], 1);
        a.slots[i] = slot;
        if (a.row_weights && slot >= 0) a.row_weights[slot] = a.weights[i];
      }
  }
}

// row t of x into the rows slots[t, 0 .. k) of out
template <typename Piece>
__global__ void __launch_bounds__(128) spread_rows_kernel(const Piece* __restrict__ x, int64_t row_x, const int32_t* __restrict__ slots, int k, int64_t pieces, Piece* __restrict__ out, int64_t out_rows) {
  griddep_launch_dependents();
  griddep_wait();
  const int64_t t = blockIdx.x;
  for (int64_t c = blockIdx.y * (int64_t)blockDim.x + threadIdx.x; c < pieces; c += (int64_t)gridDim.y * blockDim.x) {
    const Piece v = x[t * row_x + c];
    for (int j = 0; j < k; ++j) {
      const int64_t to = slots[t * k + j];
      if (to >= 0 && to < out_rows) out[to * pieces + c] = v;
    }
  }
}

struct GroupedArgs {
  const void* x;
  int x_dtype;
  int64_t x_row, x_rows;  // x's rows; row r of tile i is row i * tile + r, or, with shared rows, r
  int shared;
  const void* w;
  int w_dtype;
  int64_t w_s[3];  // matrix, row (K), column (N)
  void* out;
  int out_dtype;
  int64_t ldo, N, K;
  int tile, n;
  const int32_t *tile_expert, *live;
  const float* row_scale;
};

__device__ __forceinline__ float typed(const void* p, int dtype, int64_t at) {
  return dtype == FB_FP32 ? static_cast<const float*>(p)[at] : bf16_bits_to_float(static_cast<const uint16_t*>(p)[at]);
}

__global__ void __launch_bounds__(256) grouped_matmul_kernel(const GroupedArgs g) {
  griddep_launch_dependents();
  griddep_wait();
  const int i = blockIdx.y * 16 / g.tile, r0 = blockIdx.y * 16 % g.tile;
  if (i >= *g.live) return;
  const int e = g.tile_expert[3 * i];
  if (e < 0 || e >= g.n) return;
  __shared__ float sa[16][17], sb[16][17];
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int64_t col = blockIdx.x * 16 + tx, row = (g.shared ? 0 : (int64_t)i * g.tile) + r0 + ty, x0 = row * g.x_row;
  const bool there = row < g.x_rows;  // (a tile that holds all of a few tokens has rows to spare)
  float acc = 0.f;
  for (int64_t k0 = 0; k0 < g.K; k0 += 16) {
    sa[ty][tx] = there && k0 + tx < g.K ? typed(g.x, g.x_dtype, x0 + k0 + tx) : 0.f;
    sb[ty][tx] = col < g.N && k0 + ty < g.K ? typed(g.w, g.w_dtype, e * g.w_s[0] + (k0 + ty) * g.w_s[1] + col * g.w_s[2]) : 0.f;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) acc = fmaf(sa[ty][k], sb[k][tx], acc);
    __syncthreads();
  }
  if (col >= g.N) return;
  if (g.row_scale) acc *= g.row_scale[(int64_t)i * g.tile + r0 + ty];
  const int64_t at = ((int64_t)i * g.tile + r0 + ty) * g.ldo + col;
  if (g.out_dtype == FB_FP32) static_cast<float*>(g.out)[at] = acc;
  else static_cast<uint16_t*>(g.out)[at] = (uint16_t)float_to_bf16_bits(acc);
}

}  // namespace fb

extern "C" int64_t fb_route_tiles(int64_t T, int n, int k, int tile, int shared_rows) {
  if (T < 1 || n < 1 || k < 1 || tile < 1) return 0;
  const int64_t choices = T * k, most = choices < n ? choices : n;
  if (shared_rows) return most;
  return choices / tile + most;  // (each touched expert adds less than a tile)
}

extern "C" int fb_route(const fb_router* router_host, const float* logits, int64_t T, int64_t ld, int tile, int shared_rows, float* weights, int32_t* ids, int32_t* slots,
                        int32_t* tile_expert, int32_t* live, float* row_weights, void* stream) {
  FB_REQUIRE(router_host && logits && weights && ids && slots && tile_expert && live && T >= 1 && T <= (1 << 24), "fb_route: null pointer or no tokens");
  const int n = router_host->n, k = router_host->k, real = n - router_host->identity;
  FB_REQUIRE(router_host->identity >= 0 && real >= 1, "fb_route: at least one expert with rows");
  FB_REQUIRE(router_host->scored >= 0 && router_host->scored <= 2 && (router_host->scored || !router_host->as_scored), "fb_route: choices by logit, or scores by softmax or sigmoid, which may be the weights");
  FB_REQUIRE(n >= 1 && n <= 8192 && k >= 1 && k <= 64 && k <= n && ld >= n, "fb_route: up to 64 choices among up to 8192 experts (got %d of %d)", k, n);
  FB_REQUIRE(tile >= 16 && tile % 16 == 0 && (!shared_rows || T <= tile), "fb_route: tiles of whole runs of 16 rows; shared rows: all the tokens in one");
  const int64_t tiles = fb_route_tiles(T, real, k, tile, shared_rows);
  FB_REQUIRE(tiles * tile < (1ll << 31), "fb_route: too many rows");
  const fb::RouteArgs a{logits, T, ld, router_host->bias, n, k, tile, shared_rows, real, router_host->scored, router_host->scale, router_host->as_scored, (int)tiles, weights, ids, slots, tile_expert, live, row_weights};
  const auto s = (cudaStream_t)stream;
  const int pick = T <= 32;
  if (!pick)
    if (int rc = fb::launch_after(fb::route_tokens_kernel, dim3((unsigned)fb::ceil_div(T, 8)), dim3(256), 0, s, "fb_route", a)) return rc;
  return fb::launch_after(fb::route_places_kernel, dim3(1), dim3(1024), (size_t)(real + 33) * sizeof(int32_t), s, "fb_route", a, pick);
}

extern "C" int fb_spread_rows(const void* x, int64_t T, int64_t row_bytes, int64_t ldx_bytes, const int32_t* slots, int k, void* out, int64_t out_rows, void* stream) {
  FB_REQUIRE(x && slots && out && T >= 1 && k >= 1 && out_rows >= 1 && row_bytes >= 2 && row_bytes % 2 == 0 && ldx_bytes >= row_bytes && ldx_bytes % 2 == 0, "fb_spread_rows: null pointer, or rows of no whole 2-byte values");
  const auto s = (cudaStream_t)stream;
  if (row_bytes % 16 == 0 && ldx_bytes % 16 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)out % 16 == 0) {
    const dim3 grid((unsigned)T, (unsigned)(fb::ceil_div(row_bytes / 16, 128) < 4 ? fb::ceil_div(row_bytes / 16, 128) : 4));
    return fb::launch_after(fb::spread_rows_kernel<uint4>, grid, dim3(128), 0, s, "fb_spread_rows", (const uint4*)x, ldx_bytes / 16, slots, k, row_bytes / 16, (uint4*)out, out_rows);
  }
  return fb::launch_after(fb::spread_rows_kernel<uint16_t>, dim3((unsigned)T, 4), dim3(128), 0, s, "fb_spread_rows", (const uint16_t*)x, ldx_bytes / 2, slots, k, row_bytes / 2, (uint16_t*)out, out_rows);
}

extern "C" int fb_grouped_matmul(int x_dtype, const void* x, int64_t x_rows, int64_t ldx, int shared_rows, int w_dtype, const void* W, const int64_t* w_strides_host, int n, int64_t K, int64_t N,
                                 const int32_t* tile_expert, const int32_t* live, int64_t tiles, int tile, const float* row_scale, int out_dtype, void* out, int64_t ldo, void* stream) {
  FB_REQUIRE(x && W && w_strides_host && tile_expert && live && out && tiles >= 1 && K >= 1 && N >= 1 && n >= 1, "fb_grouped_matmul: null pointer or empty");
  FB_REQUIRE(tile >= 16 && tile % 16 == 0 && ldx >= K && ldo >= N && tiles * (tile / 16) <= 65535, "fb_grouped_matmul: tiles of whole runs of 16 rows, at most 65535 such runs");
  FB_REQUIRE(shared_rows ? x_rows >= 1 && x_rows <= tile : x_rows >= tiles * tile, "fb_grouped_matmul: all the tiles' rows there");
  for (int d : {x_dtype, w_dtype, out_dtype}) FB_REQUIRE(d == FB_BF16 || d == FB_FP32, "fb_grouped_matmul: bf16 or fp32");
  const fb::GroupedArgs g{x, x_dtype, ldx, x_rows, shared_rows, W, w_dtype, {w_strides_host[0], w_strides_host[1], w_strides_host[2]}, out, out_dtype, ldo, N, K, tile, n, tile_expert, live, row_scale};
  return fb::launch_after(fb::grouped_matmul_kernel, dim3((unsigned)fb::ceil_div(N, 16), (unsigned)(tiles * (tile / 16))), dim3(256), 0, (cudaStream_t)stream, "fb_grouped_matmul", g);
}
