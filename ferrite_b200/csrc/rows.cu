// What stands between the matmuls of a decoder with grouped-query attention and an fp32 residual stream, a kernel each:
//   fb_embed       the stream's start: a row of one table, scaled, and, where given, a row of another, added in fp32
//   fb_heads_put   after a joint q | k | v projection: biases, a short convolution over time, RMSNorm of each query and key head or
//                  of all of them together, the turn by the token's place, values mixed with another layer's or the keys
//                  themselves, the new cache row
//   fb_add_norm    a layer's end: the branches' results scaled by column, a mixture's chosen rows weighted and summed, all of that
//                  gated and normed where the design says so and added to the stream, and the next layer's RMSNorm of it
#include "launch.cuh"
#include "values.cuh"

namespace fb {

struct EmbedArgs {
  const void *table, *places_table;  // [rows, cols], [place_rows, cols] or null
  int64_t rows, place_rows, cols;
  const int32_t *ids, *places;
  float scale;
  float* out;  // [T, cols]
};

template <typename Act>
__global__ void __launch_bounds__(256) embed_kernel(const EmbedArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  const int64_t t = blockIdx.x, id = min(max((int64_t)a.ids[t], (int64_t)0), a.rows - 1);
  const Act* x = static_cast<const Act*>(a.table) + id * a.cols;
  const Act* y = nullptr;
  if (a.places_table) y = static_cast<const Act*>(a.places_table) + min(max((int64_t)a.places[t], (int64_t)0), a.place_rows - 1) * a.cols;
  for (int64_t c = threadIdx.x; c < a.cols; c += blockDim.x) a.out[t * a.cols + c] = value_of(x[c]) * a.scale + (y ? value_of(y[c]) : 0.f);
}

// ---- heads: a warp per token and head (the query heads, then the key heads, then the value heads)
struct HeadsPutArgs {
  fb_heads h;
  const void* qkv;
  int64_t T, ld;
  const int32_t* rows;
  void* q_out;
  int64_t ld_q;
  void* cache;  // [kv_heads, cache_rows, dim + vdim]: a key, then its value
  int64_t cache_rows, head_stride;
};

// what a token's queries are multiplied by after their norm
__device__ __forceinline__ float temperature_of(const fb_heads& s, int64_t t) {
  return s.temp_coef != 0.f ? fmaf(s.temp_coef, logf(floorf((float)(s.places[t] + 1) / s.temp_every) + 1.f), 1.f) : 1.f;
}

constexpr int HEADS_WARPS = 8, HEADS_REGS = 8;  // a lane keeps up to 8 columns (heads of up to 256) between the two passes

template <typename In, typename Act>
__global__ void __launch_bounds__(32 * HEADS_WARPS) heads_put_kernel(const HeadsPutArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  const fb_heads& s = a.h;
  const int lane = threadIdx.x & 31, units = s.heads + 2 * s.kv_heads;
  const int64_t t = blockIdx.x;
  const int u = blockIdx.y * HEADS_WARPS + (threadIdx.x >> 5);
  if (u >= units) return;
  const bool is_q = u < s.heads, is_v = u >= s.heads + s.kv_heads;
  const int n = is_v ? s.vdim : s.dim, g = is_q ? u : is_v ? u - s.heads - s.kv_heads : u - s.heads;
  const int64_t at = is_v ? (int64_t)(s.heads + s.kv_heads) * s.dim + (int64_t)g * s.vdim : (int64_t)u * s.dim;
  const int64_t row = a.rows[t];
  if (!is_q && (row < 0 || row >= a.cache_rows)) return;  // nothing is written outside the cache
  const In* x = static_cast<const In*>(a.qkv) + t * a.ld + at;
  const float* bias = s.bias ? s.bias + at : nullptr;
  Act* out = is_q ? static_cast<Act*>(a.q_out) + t * a.ld_q + (int64_t)g * s.dim
                  : static_cast<Act*>(a.cache) + g * a.head_stride + row * (s.dim + s.vdim) + (is_v ? s.dim : 0);
  if (is_v) {
    const In* first = s.first ? static_cast<const In*>(s.first) + t * s.ld_first + (int64_t)g * s.vdim : nullptr;
    const float* first_bias = s.first && s.first_bias ? s.first_bias + (int64_t)g * s.vdim : nullptr;
    const float share = s.first ? *s.share : 0.f;
    for (int c = lane; c < n; c += 32) {
      float v = value_of(x[c]) + (bias ? bias[c] : 0.f);
      if (first) v = (1.f - share) * v + share * (value_of(first[c]) + (first_bias ? first_bias[c] : 0.f));
      store_value(out + c, v);
    }
    return;
  }
  const float* w = is_q ? s.q_norm : s.k_norm;
  float keep[HEADS_REGS], ss = 0.f;
#pragma unroll
  for (int i = 0; i < HEADS_REGS; ++i) {
    const int c = 32 * i + lane;
    keep[i] = c < n ? value_of(x[c]) + (bias ? bias[c] : 0.f) : 0.f;
    ss = fmaf(keep[i], keep[i], ss);
  }
  for (int c = 32 * HEADS_REGS + lane; c < n; c += 32) {  // (wider heads: read twice)
    const float v = value_of(x[c]) + (bias ? bias[c] : 0.f);
    ss = fmaf(v, v, ss);
  }
  const float r = (w ? 1.f / sqrtf(warp_sum(ss) / (float)n + s.eps) : 1.f) * (is_q ? temperature_of(s, t) : 1.f);
#pragma unroll
  for (int i = 0; i < HEADS_REGS; ++i) {
    const int c = 32 * i + lane;
    if (c < n) store_value(out + c, keep[i] * r * (w ? w[c] : 1.f));
  }
  for (int c = 32 * HEADS_REGS + lane; c < n; c += 32) store_value(out + c, (value_of(x[c]) + (bias ? bias[c] : 0.f)) * r * (w ? w[c] : 1.f));
}

// the same for heads of whole groups of four columns, 16-byte aligned, up to 256 wide: a warp has four heads, everything it
// reads on its way at once
template <typename In, typename Act, int GROUPS>
__global__ void __launch_bounds__(128) heads_put4_kernel(const HeadsPutArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  constexpr int UNITS = 4;
  const fb_heads& s = a.h;
  const int lane = threadIdx.x & 31, keys = s.heads + s.kv_heads, units = keys + s.kv_heads;
  const int64_t t = blockIdx.x, row = a.rows[t];
  const bool inside = row >= 0 && row < a.cache_rows;  // nothing is written outside the cache
  const int u0 = (blockIdx.y * 4 + (threadIdx.x >> 5)) * UNITS;
  const In* x = static_cast<const In*>(a.qkv) + t * a.ld;
  float4 v[UNITS][GROUPS], f[UNITS][GROUPS];
#pragma unroll
  for (int i = 0; i < UNITS; ++i)
#pragma unroll
    for (int j = 0; j < GROUPS; ++j) {
      const int u = u0 + i, c = 4 * (32 * j + lane);
      v[i][j] = f[i][j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (u >= units || c >= (u < keys ? s.dim : s.vdim)) continue;
      const int64_t at = u < keys ? (int64_t)u * s.dim : (int64_t)keys * s.dim + (int64_t)(u - keys) * s.vdim;
      v[i][j] = four(x + at + c);
      if (u >= keys && s.first) f[i][j] = four(static_cast<const In*>(s.first) + t * s.ld_first + (int64_t)(u - keys) * s.vdim + c);
    }
  const float share = s.first ? *s.share : 0.f, temp = temperature_of(s, t);
#pragma unroll
  for (int i = 0; i < UNITS; ++i) {
    const int u = u0 + i, n = u < keys ? s.dim : s.vdim;
    if (u >= units) break;
    const int64_t at = u < keys ? (int64_t)u * s.dim : (int64_t)keys * s.dim + (int64_t)(u - keys) * s.vdim;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < GROUPS; ++j) {
      const int c = 4 * (32 * j + lane);
      if (c < n && s.bias) {
        const float4 b = four(s.bias + at + c);
        v[i][j].x += b.x, v[i][j].y += b.y, v[i][j].z += b.z, v[i][j].w += b.w;
      }
      if (u >= keys && s.first && c < n) {
        float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s.first_bias) b = four(s.first_bias + (int64_t)(u - keys) * s.vdim + c);
        v[i][j].x = (1.f - share) * v[i][j].x + share * (f[i][j].x + b.x), v[i][j].y = (1.f - share) * v[i][j].y + share * (f[i][j].y + b.y);
        v[i][j].z = (1.f - share) * v[i][j].z + share * (f[i][j].z + b.z), v[i][j].w = (1.f - share) * v[i][j].w + share * (f[i][j].w + b.w);
      }
      ss = fmaf(v[i][j].x, v[i][j].x, fmaf(v[i][j].y, v[i][j].y, fmaf(v[i][j].z, v[i][j].z, fmaf(v[i][j].w, v[i][j].w, ss))));
    }
    const float* w = u < s.heads ? s.q_norm : u < keys ? s.k_norm : nullptr;
    const float r = (w ? 1.f / sqrtf(warp_sum(ss) / (float)n + s.eps) : 1.f) * (u < s.heads ? temp : 1.f);
    if (u >= s.heads && !inside) continue;
    Act* out = u < s.heads ? static_cast<Act*>(a.q_out) + t * a.ld_q + (int64_t)u * s.dim
                           : static_cast<Act*>(a.cache) + (u < keys ? u - s.heads : u - keys) * a.head_stride + row * (s.dim + s.vdim) + (u < keys ? 0 : s.dim);
#pragma unroll
    for (int j = 0; j < GROUPS; ++j) {
      const int c = 4 * (32 * j + lane);
      if (c >= n) continue;
      const float4 g = w ? four(w + c) : make_float4(1.f, 1.f, 1.f, 1.f);
      put_four(out + c, make_float4(v[i][j].x * r * g.x, v[i][j].y * r * g.y, v[i][j].z * r * g.z, v[i][j].w * r * g.w));
    }
  }
}

// ---- the same with a convolution, joint norms, turned heads or keys that are the values too: a block has a token's units - all
// query heads, or the others, where a norm goes over them together; else some of them - and keeps their columns in shared memory.
// The tokens whose convolution reaches into the state are one block's, one after the other, which then leaves the new state: no
// other block reads or writes it.
struct HeadsTurnArgs {
  HeadsPutArgs p;
  int per, tokens, first, group;  // units a block (joint norms: 0); tokens of a sequence, how many of them its first block has, and each other
};

// N values at p
template <int N, typename T>
__device__ __forceinline__ void read_some(const T* p, float v[N]) {
  if constexpr (N == 4) {
    const float4 f = four(p);
    v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
  } else {
    v[0] = value_of(p[0]);
  }
}
template <int N, typename T>
__device__ __forceinline__ void put_some(T* p, const float v[N]) {
  if constexpr (N == 4) put_four(p, make_float4(v[0], v[1], v[2], v[3]));
  else store_value(p, v[0]);
}

template <typename In, typename Act, int N>  // N: columns a thread handles at a time, 4 (whole aligned groups) or 1
__global__ void __launch_bounds__(512) heads_turn_kernel(const HeadsTurnArgs args) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ __align__(16) float turn_row[];  // the block's columns, then [turned / 2] cos and sin
  __shared__ float red[32];
  const HeadsPutArgs& a = args.p;
  const fb_heads& s = a.h;
  const int keys = s.heads + s.kv_heads, units = s.keys_are_values ? keys : keys + s.kv_heads;
  const int u0 = args.per ? blockIdx.y * args.per : blockIdx.y ? s.heads : 0, u1 = args.per ? min(units, u0 + args.per) : blockIdx.y ? units : s.heads;
  auto column = [&](int u) { return min(u, keys) * s.dim + max(u - keys, 0) * s.vdim; };  // (fewer than 2^30 columns, the caller has seen to it)
  const int c0 = column(u0), all = column(units), cols = column(u1) - c0, key_cols = column(keys) - c0;
  float *turns = turn_row + (cols + 3) / 4 * 4;
  const int half = s.turned / 2, blocks = 1 + (args.tokens - args.first + args.group - 1) / args.group;
  const int seq = blockIdx.x / blocks, b = blockIdx.x % blocks, begin = b ? args.first + (b - 1) * args.group : 0, count = b ? min(args.group, args.tokens - begin) : args.first;
  const int64_t row0 = (int64_t)seq * args.tokens;
  const int start = s.places ? s.places[row0] : 0;  // where the sequence's first token of this call stands
  const bool dead = s.conv && start == s.dead, held = s.conv && start != 0 && !dead;
  const int back = s.conv ? s.taps - 1 : 0;
  const In* x = static_cast<const In*>(a.qkv) + row0 * a.ld + c0;
  float* state = s.conv ? s.state + seq * s.state_stride + c0 : nullptr;
  // N columns of the sequence's token i as projected, from the state where i < 0
  auto projected = [&](int i, int c, float v[N]) {
    if (i >= 0) {
      read_some<N>(x + (int64_t)i * a.ld + c, v);
      if (s.bias) {
        float bias[N];
        read_some<N>(s.bias + c0 + c, bias);
#pragma unroll
        for (int e = 0; e < N; ++e) v[e] += bias[e];
      }
    } else {
#pragma unroll
      for (int e = 0; e < N; ++e) v[e] = held ? state[(int64_t)(back + i) * all + c + e] : 0.f;
    }
  };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = begin; i < begin + count; ++i) {
    const int64_t t = row0 + i, row = a.rows[t];
    if (s.turned) {
      const int place = s.places[t];
      for (int j = threadIdx.x; j < half; j += blockDim.x) turn_of(place, s.freq[j], s.mag, turns[j], turns[half + j]);
    }
    float ss = 0.f;
    for (int c = N * threadIdx.x; c < cols; c += N * blockDim.x) {
      float v[N];
      if (s.conv) {
#pragma unroll
        for (int e = 0; e < N; ++e) v[e] = 0.f;
#pragma unroll 4
        for (int j = 0; j < s.taps; ++j) {
          float u[N], weight[N];
          projected(i - back + j, c, u);
          read_some<N>(s.conv + j * all + c0 + c, weight);
#pragma unroll
          for (int e = 0; e < N; ++e) v[e] = fmaf(weight[e], u[e], v[e]);
        }
      } else {
        projected(i, c, v);
      }
#pragma unroll
      for (int e = 0; e < N; ++e)
        if (s.norm_all && c + e < key_cols) ss = fmaf(v[e], v[e], ss);  // (a block's query heads, or its key heads)
      put_some<N>(turn_row + c, v);
    }
    const float joint = s.norm_all ? 1.f / sqrtf(block_sum(ss, red) / (float)((blockIdx.y ? s.kv_heads : s.heads) * s.dim) + s.eps) : 1.f;
    __syncthreads();
    const bool inside = row >= 0 && row < a.cache_rows;  // nothing is written outside the cache
    const float temp = temperature_of(s, t);
    for (int u = u0 + warp; u < u1; u += blockDim.x / 32) {
      const bool is_q = u < s.heads, is_v = u >= keys;
      const int n = is_v ? s.vdim : s.dim, g = is_q ? u : is_v ? u - keys : u - s.heads;
      if (!is_q && !inside) continue;
      const float* mine = turn_row + (column(u) - c0);
      const float* w = is_v ? nullptr : is_q ? s.q_norm : s.k_norm;
      if (w && s.norm_all) w += g * s.dim;
      float r = joint;
      if (w && !s.norm_all) {
        float own = 0.f;
        for (int c = lane; c < n; c += 32) own = fmaf(mine[c], mine[c], own);
        r = 1.f / sqrtf(warp_sum(own) / (float)n + s.eps);
      }
      Act* cached = static_cast<Act*>(a.cache) + g * a.head_stride + row * (s.dim + s.vdim);
      Act* out = is_q ? static_cast<Act*>(a.q_out) + t * a.ld_q + (int64_t)g * s.dim : is_v ? cached + s.dim : cached;
      for (int c = N * lane; c < n; c += 32 * N) {
        float v[N];
        read_some<N>(mine + c, v);
        if (s.keys_are_values && !is_q) put_some<N>(cached + s.dim + c, v);
        if (w) {
          float g4[N];
          read_some<N>(w + c, g4);
#pragma unroll
          for (int e = 0; e < N; ++e) v[e] *= r * g4[e];
        }
        if (is_q) {
#pragma unroll
          for (int e = 0; e < N; ++e) v[e] *= temp;
        }
        if (!is_v && c < s.turned) {
          if constexpr (N == 4) {
#pragma unroll
            for (int e = 0; e < 4; e += 2)
              if (c + e < s.turned) {
                const float cs = turns[(c + e) / 2], sn = turns[half + (c + e) / 2], x0 = v[e], x1 = v[e + 1];
                v[e] = x0 * cs - x1 * sn, v[e + 1] = x1 * cs + x0 * sn;
              }
          } else {
            const float other = mine[c ^ 1] * (w ? r * w[c ^ 1] : 1.f) * (is_q ? temp : 1.f), cs = turns[c >> 1], sn = turns[half + (c >> 1)];
            v[0] = c & 1 ? v[0] * cs + other * sn : v[0] * cs - other * sn;
          }
        }
        put_some<N>(out + c, v);
      }
    }
    __syncthreads();
  }
  if (s.conv && b == 0 && !dead)  // (a thread's own columns, rows rising: what a row is made of is read before it is overwritten)
    for (int c = N * threadIdx.x; c < cols; c += N * blockDim.x)
      for (int r = 0; r < back; ++r) {
        float v[N];
        projected(args.tokens + r - back, c, v);
#pragma unroll
        for (int e = 0; e < N; ++e) state[r * all + c + e] = v[e];
      }
}

template <typename In, typename Act>
static int launch_heads_turn(const HeadsPutArgs& a, cudaStream_t s) {
  const fb_heads& h = a.h;
  HeadsTurnArgs t{a, 0, 1, 1, 1};
  const int units = h.heads + (h.keys_are_values ? 1 : 2) * h.kv_heads, wide = h.dim > h.vdim ? h.dim : h.vdim;
  unsigned parts = 2;
  int64_t most = (int64_t)(h.heads > 2 * h.kv_heads ? h.heads : 2 * h.kv_heads) * wide;
  if (!h.norm_all) {
    t.per = 1024 / wide < 1 ? 1 : 1024 / wide;
    parts = (unsigned)ceil_div(units, t.per), most = (int64_t)t.per * wide;
  }
  const size_t smem = (size_t)((most + 3) / 4 * 4 + h.turned) * sizeof(float);
  FB_REQUIRE(smem <= 200 * 1024, "fb_heads_put: too many columns for a norm over all heads");
  int64_t grid = a.T;
  if (h.conv) {
    t.tokens = (int)(a.T / h.sequences), t.first = h.taps - 1 < 1 ? 1 : h.taps - 1 < t.tokens ? h.taps - 1 : t.tokens;
    while (t.group < 8 && ceil_div(a.T, 2 * t.group) * parts >= 8 * 148) t.group *= 2;  // (a block's next token finds the weights and the rows before it near)
    grid = (int64_t)h.sequences * (1 + ceil_div(t.tokens - t.first, t.group));
  }
  auto whole = [](const void* p, int64_t ld, int bytes) { return (uintptr_t)p % (4 * bytes) == 0 && ld % 4 == 0; };
  const bool fours = h.dim % 4 == 0 && h.vdim % 4 == 0 && whole(a.qkv, a.ld, sizeof(In)) && whole(a.q_out, a.ld_q, sizeof(Act)) && whole(a.cache, a.head_stride, sizeof(Act)) &&
                     whole(h.bias, 0, 4) && whole(h.conv, 0, 4) && whole(h.q_norm, 0, 4) && whole(h.k_norm, 0, 4);
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) {
    cudaFuncSetAttribute(heads_turn_kernel<In, Act, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    cudaFuncSetAttribute(heads_turn_kernel<In, Act, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  }
  const dim3 g((unsigned)grid, parts), block(most > 1024 && h.norm_all ? 512 : 256);
  return fours ? launch_after(heads_turn_kernel<In, Act, 4>, g, block, smem, s, "fb_heads_put", t) : launch_after(heads_turn_kernel<In, Act, 1>, g, block, smem, s, "fb_heads_put", t);
}

template <typename In, typename Act>
static int launch_heads_put(const HeadsPutArgs& a, cudaStream_t s) {
  const fb_heads& h = a.h;
  if (h.turned || h.conv || h.norm_all || h.keys_are_values) return launch_heads_turn<In, Act>(a, s);
  const int units = h.heads + 2 * h.kv_heads;
  auto whole = [](const void* p, int64_t ld, int bytes) { return (uintptr_t)p % (4 * bytes) == 0 && ld % 4 == 0; };
  const bool fours = h.dim % 4 == 0 && h.vdim % 4 == 0 && h.dim <= 256 && h.vdim <= 256 && whole(a.qkv, a.ld, sizeof(In)) && whole(h.first, h.ld_first, sizeof(In)) && whole(h.bias, 0, 4) &&
                     whole(h.first_bias, 0, 4) && whole(h.q_norm, 0, 4) && whole(h.k_norm, 0, 4) && whole(a.q_out, a.ld_q, sizeof(Act)) && whole(a.cache, a.head_stride, sizeof(Act));
  if (fours) {
    const dim3 grid((unsigned)a.T, (unsigned)ceil_div(units, 16));
    if (h.dim <= 128 && h.vdim <= 128) return launch_after(heads_put4_kernel<In, Act, 1>, grid, dim3(128), 0, s, "fb_heads_put", a);
    return launch_after(heads_put4_kernel<In, Act, 2>, grid, dim3(128), 0, s, "fb_heads_put", a);
  }
  return launch_after(heads_put_kernel<In, Act>, dim3((unsigned)a.T, (unsigned)ceil_div(units, HEADS_WARPS)), dim3(32 * HEADS_WARPS), 0, s, "fb_heads_put", a);
}

// where a token's chosen rows are: one with slot -1 is the token's own (or, where there are none, counts for nothing)
template <typename Act>
__device__ __forceinline__ void chosen_rows(const fb_branches& a, int64_t t, const Act** from, float* weight) {
  for (int j = threadIdx.x; j < a.k; j += blockDim.x) {
    const int64_t slot = a.slots[t * a.k + j];
    const bool own = slot < 0 && a.own;
    from[j] = own ? static_cast<const Act*>(a.own) + t * a.ld_own : static_cast<const Act*>(a.chosen) + (slot < 0 ? 0 : slot) * a.ld_chosen;
    weight[j] = slot < 0 && !own ? 0.f : a.weights ? a.weights[t * a.k + j] : 1.f;
  }
}

// ---- a layer's end: a block per token; the new row stays in shared memory for the norm's second pass
template <typename In, typename Act>
__global__ void __launch_bounds__(512) add_norm_kernel(const fb_branches a, const int64_t cols) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ float row[];  // [cols]
  __shared__ float red[32];
  __shared__ const Act* from[64];
  __shared__ float weight[64];
  const int64_t t = blockIdx.x;
  if (a.chosen) chosen_rows(a, t, from, weight);
  __syncthreads();
  const float* x = a.x + t * a.ld_x;
  const In* y1 = a.mixer ? static_cast<const In*>(a.mixer) + t * a.ld_mixer : nullptr;
  const In* y2 = a.other ? static_cast<const In*>(a.other) + t * a.ld_other : nullptr;
  const bool apart = a.gate || a.post;  // the branches' sum is finished before the stream joins
  float ss = 0.f;
  for (int64_t c = threadIdx.x; c < cols; c += blockDim.x) {
    float v = apart ? 0.f : x[c];
    if (y1 || a.mixer_bias) v = fmaf((y1 ? value_of(y1[c]) : 0.f) + (a.mixer_bias ? a.mixer_bias[c] : 0.f), a.mixer_scale ? a.mixer_scale[c] : 1.f, v);
    if (a.chosen || y2) {
      float f = y2 ? value_of(y2[c]) : 0.f;
      if (a.chosen)
        for (int j = 0; j < a.k; ++j) f = fmaf(weight[j], value_of(from[j][c]), f);
      v = fmaf(f, a.other_scale ? a.other_scale[c] : 1.f, v);
    }
    if (a.gate) v *= sigmoid_f(a.gate[t * a.ld_gate + c] + (a.gate_bias ? a.gate_bias[c] : 0.f));
    row[c] = v;
    if (a.x_out && !apart) a.x_out[t * a.ld_x_out + c] = v;
    ss = fmaf(v, v, ss);
  }
  if (apart) {
    const float r = a.post ? 1.f / sqrtf(block_sum(ss, red) / (float)cols + a.eps) : 1.f;
    ss = 0.f;
    for (int64_t c = threadIdx.x; c < cols; c += blockDim.x) {
      const float v = fmaf(row[c] * r, a.post ? a.post[c] : 1.f, x[c]);
      row[c] = v;
      if (a.x_out) a.x_out[t * a.ld_x_out + c] = v;
      ss = fmaf(v, v, ss);
    }
  }
  if (!a.h) return;
  const float r = a.w ? 1.f / sqrtf(block_sum(ss, red) / (float)cols + a.eps) : 1.f;
  Act* h = static_cast<Act*>(a.h) + t * a.ld_h;
  for (int64_t c = threadIdx.x; c < cols; c += blockDim.x) store_value(h + c, a.w ? row[c] * r * (a.w[c] + a.plus) : row[c]);
}

// the same for rows of whole groups of four columns, 16-byte aligned: a thread keeps its groups in registers, everything it
// reads on its way at once
template <typename In, typename Act, int GROUPS, bool APART>
__global__ void __launch_bounds__(512) add_norm4_kernel(const fb_branches a, const int64_t cols) {
  griddep_launch_dependents();
  griddep_wait();
  __shared__ float red[32];
  __shared__ const Act* from[64];
  __shared__ float weight[64];
  const int64_t t = blockIdx.x;
  if (a.chosen) {
    chosen_rows(a, t, from, weight);
    __syncthreads();
  }
  const float4 one = make_float4(1.f, 1.f, 1.f, 1.f), none = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 v[GROUPS], f[GROUPS], x[APART ? GROUPS : 1], gate[APART ? GROUPS : 1];  // APART: the branches' sum is finished before the stream joins
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < GROUPS; ++i) {
    const int64_t c = 4 * (threadIdx.x + (int64_t)i * blockDim.x);
    v[i] = f[i] = none;
    if (c >= cols) continue;
    if constexpr (APART) {
      x[i] = four(a.x + t * a.ld_x + c), gate[i] = none;
      if (a.gate) gate[i] = four(a.gate + t * a.ld_gate + c);
    } else {
      v[i] = four(a.x + t * a.ld_x + c);
    }
    if (a.mixer) v[i] = fma4(four(static_cast<const In*>(a.mixer) + t * a.ld_mixer + c), a.mixer_scale ? four(a.mixer_scale + c) : one, v[i]);
    if (a.mixer_bias) v[i] = fma4(four(a.mixer_bias + c), a.mixer_scale ? four(a.mixer_scale + c) : one, v[i]);
    if (a.other) f[i] = four(static_cast<const In*>(a.other) + t * a.ld_other + c);
  }
  if (a.chosen)
    for (int j = 0; j < a.k; j += 4) {
      float4 part[GROUPS][4];
#pragma unroll
      for (int i = 0; i < GROUPS; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int64_t c = 4 * (threadIdx.x + (int64_t)i * blockDim.x);
          part[i][e] = j + e < a.k && c < cols ? four(from[j + e] + c) : none;
        }
#pragma unroll
      for (int i = 0; i < GROUPS; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float s = j + e < a.k ? weight[j + e] : 0.f;
          f[i] = fma4(make_float4(s, s, s, s), part[i][e], f[i]);
        }
    }
#pragma unroll
  for (int i = 0; i < GROUPS; ++i) {
    const int64_t c = 4 * (threadIdx.x + (int64_t)i * blockDim.x);
    if (c >= cols) continue;
    if (a.chosen || a.other) v[i] = fma4(f[i], a.other_scale ? four(a.other_scale + c) : one, v[i]);
    if constexpr (APART) {
      if (a.gate) {
        const float4 b = a.gate_bias ? four(a.gate_bias + c) : none;
        v[i].x *= sigmoid_f(gate[i].x + b.x), v[i].y *= sigmoid_f(gate[i].y + b.y), v[i].z *= sigmoid_f(gate[i].z + b.z), v[i].w *= sigmoid_f(gate[i].w + b.w);
      }
      ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
      continue;
    }
    if (a.x_out) put_four(a.x_out + t * a.ld_x_out + c, v[i]);
    ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
  }
  if constexpr (APART) {
    const float r = a.post ? 1.f / sqrtf(block_sum(ss, red) / (float)cols + a.eps) : 1.f;
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < GROUPS; ++i) {
      const int64_t c = 4 * (threadIdx.x + (int64_t)i * blockDim.x);
      if (c >= cols) continue;
      v[i] = fma4(make_float4(v[i].x * r, v[i].y * r, v[i].z * r, v[i].w * r), a.post ? four(a.post + c) : one, x[i]);
      if (a.x_out) put_four(a.x_out + t * a.ld_x_out + c, v[i]);
      ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
    }
  }
  if (!a.h) return;
  const float r = a.w ? 1.f / sqrtf(block_sum(ss, red) / (float)cols + a.eps) : 1.f;
#pragma unroll
  for (int i = 0; i < GROUPS; ++i) {
    const int64_t c = 4 * (threadIdx.x + (int64_t)i * blockDim.x);
    if (c >= cols) continue;
    if (!a.w) {
      put_four(static_cast<Act*>(a.h) + t * a.ld_h + c, v[i]);
      continue;
    }
    const float4 w = four(a.w + c);
    put_four(static_cast<Act*>(a.h) + t * a.ld_h + c,
             make_float4(v[i].x * r * (w.x + a.plus), v[i].y * r * (w.y + a.plus), v[i].z * r * (w.z + a.plus), v[i].w * r * (w.w + a.plus)));
  }
}

template <typename In, typename Act, int GROUPS>
static int launch_add_norm4(const fb_branches& a, int64_t T, dim3 block, int64_t cols, cudaStream_t s) {
  if (a.gate || a.post) return launch_after(add_norm4_kernel<In, Act, GROUPS, true>, dim3((unsigned)T), block, 0, s, "fb_add_norm", a, cols);
  return launch_after(add_norm4_kernel<In, Act, GROUPS, false>, dim3((unsigned)T), block, 0, s, "fb_add_norm", a, cols);
}

template <typename In, typename Act>
static int launch_add_norm(const fb_branches& a, int64_t T, int64_t cols, cudaStream_t s) {
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(add_norm_kernel<In, Act>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  auto whole = [](const void* p, int64_t ld, int bytes) { return (uintptr_t)p % (4 * bytes) == 0 && ld % 4 == 0; };
  const bool fours = cols % 4 == 0 && cols <= 4 * 4 * 512 && whole(a.x, a.ld_x, 4) && whole(a.mixer, a.ld_mixer, sizeof(In)) && whole(a.mixer_scale, 0, 4) &&
                     whole(a.other, a.ld_other, sizeof(In)) && whole(a.other_scale, 0, 4) && whole(a.chosen, a.ld_chosen, sizeof(Act)) && whole(a.x_out, a.ld_x_out, 4) && whole(a.w, 0, 4) && whole(a.mixer_bias, 0, 4) && whole(a.own, a.ld_own, sizeof(Act)) && whole(a.gate, a.ld_gate, 4) &&
                     whole(a.gate_bias, 0, 4) && whole(a.post, 0, 4) &&
                     whole(a.h, a.ld_h, sizeof(Act));
  const dim3 grid((unsigned)T);
  auto warps = [](int64_t work) { return dim3((unsigned)(work >= 512 ? 512 : ceil_div(work, 32) * 32)); };
  if (!fours) return launch_after(add_norm_kernel<In, Act>, grid, warps(cols), (size_t)cols * sizeof(float), s, "fb_add_norm", a, cols);
  // few rows: a thread a group of four columns; many: fewer threads with more on their way each
  const int groups = cols > 4 * 1024 ? 4 : cols > 4 * 512 || T >= 512 ? 2 : 1;
  const dim3 block = warps(ceil_div(cols / 4, groups));
  if (groups == 4) return launch_add_norm4<In, Act, 4>(a, T, block, cols, s);
  if (groups == 2) return launch_add_norm4<In, Act, 2>(a, T, block, cols, s);
  return launch_add_norm4<In, Act, 1>(a, T, block, cols, s);
}

}  // namespace fb

extern "C" int fb_embed(int dtype, const void* table, int64_t rows, int64_t cols, const int32_t* ids, const void* places_table, int64_t place_rows, const int32_t* places,
                        int64_t T, float scale, float* out, void* stream) {
  FB_REQUIRE(table && ids && out && T >= 1 && rows >= 1 && cols >= 1, "fb_embed: null pointer or empty");
  FB_REQUIRE(!places_table || (places && place_rows >= 1), "fb_embed: a table of places takes the places");
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "fb_embed: bf16 or fp32 tables");
  const fb::EmbedArgs a{table, places_table, rows, place_rows, cols, ids, places, scale, out};
  const auto s = (cudaStream_t)stream;
  if (dtype == FB_FP32) return fb::launch_after(fb::embed_kernel<float>, dim3((unsigned)T), dim3(256), 0, s, "fb_embed", a);
  return fb::launch_after(fb::embed_kernel<uint16_t>, dim3((unsigned)T), dim3(256), 0, s, "fb_embed", a);
}

extern "C" int fb_heads_put(const fb_heads* heads_host, int in_dtype, const void* qkv, int64_t T, int64_t ld, const int32_t* rows, int dtype, void* q_out, int64_t ld_q,
                            void* cache, int64_t cache_rows, int64_t head_stride, void* stream) {
  FB_REQUIRE(heads_host && qkv && rows && q_out && cache && T >= 1, "fb_heads_put: null pointer or empty");
  const fb_heads& h = *heads_host;
  FB_REQUIRE(h.heads >= 1 && h.kv_heads >= 1 && h.heads % h.kv_heads == 0 && h.heads <= 100000 && h.dim >= 1 && h.vdim >= 1, "fb_heads_put: whole groups of query heads per key head (got %d / %d)", h.heads, h.kv_heads);
  const int64_t cols = (int64_t)(h.heads + h.kv_heads) * h.dim + (h.keys_are_values ? 0 : (int64_t)h.kv_heads * h.vdim);
  FB_REQUIRE(cols < (1 << 30), "fb_heads_put: too many columns");
  FB_REQUIRE(!h.keys_are_values || h.vdim == h.dim, "fb_heads_put: values that are keys are as wide");
  FB_REQUIRE(h.turned >= 0 && h.turned % 2 == 0 && h.turned <= h.dim && (!h.turned || (h.freq && h.places)), "fb_heads_put: an even number of a head's columns turn, by frequencies and places");
  FB_REQUIRE(!h.conv || (h.taps >= 1 && h.state && h.places && h.sequences >= 1 && T % h.sequences == 0 && (h.sequences == 1 || h.state_stride >= (h.taps - 1) * cols)),
             "fb_heads_put: a convolution takes its state, the places, and as many rows of each sequence");
  FB_REQUIRE(h.temp_coef == 0.f || (h.places && h.temp_every > 0.f), "fb_heads_put: a temperature by place takes the places and a positive step");
  FB_REQUIRE(!h.norm_all || (h.q_norm && h.k_norm), "fb_heads_put: a norm over all heads takes its weights");
  FB_REQUIRE(!h.first || !(h.turned || h.conv || h.norm_all || h.keys_are_values), "fb_heads_put: mixed values go with plain heads");
  FB_REQUIRE(ld >= cols && ld_q >= (int64_t)h.heads * h.dim && cache_rows >= 1 && head_stride >= cache_rows * (h.dim + h.vdim), "fb_heads_put: row strides too small");
  FB_REQUIRE(!h.first || (h.share && h.ld_first >= (int64_t)h.kv_heads * h.vdim), "fb_heads_put: mixed values take the other layer's and their share");
  FB_REQUIRE((in_dtype == FB_BF16 || in_dtype == FB_FP32) && (dtype == FB_BF16 || dtype == FB_FP32) && (in_dtype == FB_FP32 || dtype == FB_BF16),
             "fb_heads_put: bf16 or fp32; fp32 results come from fp32");
  const fb::HeadsPutArgs a{h, qkv, T, ld, rows, q_out, ld_q, cache, cache_rows, head_stride};
  const auto s = (cudaStream_t)stream;
  if (in_dtype == FB_FP32 && dtype == FB_FP32) return fb::launch_heads_put<float, float>(a, s);
  if (in_dtype == FB_FP32) return fb::launch_heads_put<float, uint16_t>(a, s);
  return fb::launch_heads_put<uint16_t, uint16_t>(a, s);
}

extern "C" int fb_add_norm(const fb_branches* branches_host, int64_t T, int64_t cols, int in_dtype, int dtype, void* stream) {
  FB_REQUIRE(branches_host && branches_host->x && T >= 1 && cols >= 1 && cols * 4 <= 200 * 1024, "fb_add_norm: null pointer, empty or rows past 51200 columns");
  const fb_branches& a = *branches_host;
  FB_REQUIRE(a.x_out || a.h, "fb_add_norm: no result");
  FB_REQUIRE(!a.gate || a.ld_gate >= cols, "fb_add_norm: a gate a column");
  FB_REQUIRE(!a.chosen || (a.slots && a.k >= 1 && a.k <= 64), "fb_add_norm: chosen rows take their places, up to 64 a token");
  FB_REQUIRE((in_dtype == FB_BF16 || in_dtype == FB_FP32) && (dtype == FB_BF16 || dtype == FB_FP32) && (in_dtype == FB_FP32 || dtype == FB_BF16),
             "fb_add_norm: bf16 or fp32; fp32 results come from fp32");
  const auto s = (cudaStream_t)stream;
  if (in_dtype == FB_FP32 && dtype == FB_FP32) return fb::launch_add_norm<float, float>(a, T, cols, s);
  if (in_dtype == FB_FP32) return fb::launch_add_norm<float, uint16_t>(a, T, cols, s);
  return fb::launch_add_norm<uint16_t, uint16_t>(a, T, cols, s);
}
