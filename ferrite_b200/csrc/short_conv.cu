// Short convolutions over time, and the gated linear recurrence that follows one:
//   fb_short_conv   y_t = bias + sum_j w_j x_(t - taps + 1 + j) per column, then SiLU where asked for; a sequence's last taps - 1
//                   inputs are kept in fp32 for the next call
//   fb_lru_scan     S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t per column, a_t = exp(rate r_t softplus(lam)), r and i sigmoids of
//                   gates; times the GELU of another branch.  One token a sequence: a thread a column.  A prompt: a CTA has 16
//                   columns; 32 runs of 8 tokens go side by side, each from zero, and meet by their products of a
#include "launch.cuh"
#include "values.cuh"

namespace fb {

struct ConvArgs {
  fb_conv c;
  const void* x;
  int64_t ld;
  void* out;
  int64_t ld_o;
  int first, group;  // tokens that a sequence's first block has - those whose sum reaches into the state -, and each other
};

template <int N, typename T>
__device__ __forceinline__ void get_some(const T* p, float v[N]) {
  if constexpr (N == 4) {
    const float4 f = four(p);
    v[0] = f.x, v[1] = f.y, v[2] = f.z, v[3] = f.w;
  } else {
    v[0] = value_of(p[0]);
  }
}
template <int N, typename T>
__device__ __forceinline__ void set_some(T* p, const float v[N]) {
  if constexpr (N == 4) put_four(p, make_float4(v[0], v[1], v[2], v[3]));
  else store_value(p, v[0]);
}

constexpr int CONV_THREADS = 128, CONV_KEPT = 4, CONV_AHEAD = 2;  // up to CONV_KEPT taps the inputs go through registers, each read once a block

// A block has N columns a thread and a run of one sequence's tokens.  The first run's block alone reads and leaves the state.
template <typename In, typename Act, int N, int TAPS>  // TAPS 0: any number, inputs read anew for every token
__global__ void __launch_bounds__(CONV_THREADS) short_conv_kernel(const ConvArgs args) {
  griddep_launch_dependents();
  griddep_wait();
  const fb_conv& a = args.c;
  const int64_t col = ((int64_t)blockIdx.y * CONV_THREADS + threadIdx.x) * N;
  if (col >= a.cols) return;
  const int64_t blocks = 1 + (a.tokens - args.first + args.group - 1) / args.group;
  const int64_t seq = blockIdx.x / blocks, b = blockIdx.x % blocks, begin = b ? args.first + (b - 1) * args.group : 0, end = b ? min(a.tokens, begin + args.group) : args.first;
  const int64_t row0 = seq * a.tokens;
  const int taps = TAPS ? TAPS : a.taps, back = taps - 1, start = a.places[row0];
  const bool dead = start == a.dead, held = start != 0 && !dead;
  const In* x = static_cast<const In*>(args.x) + row0 * args.ld + col;
  float* state = a.state ? a.state + seq * a.state_stride + col : nullptr;
  float in_bias[N], bias[N], own[TAPS ? TAPS : 1][N];
#pragma unroll
  for (int e = 0; e < N; ++e) in_bias[e] = a.in_bias ? a.in_bias[col + e] : 0.f, bias[e] = a.bias ? a.bias[col + e] : 0.f;
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) get_some<N>(a.w + j * a.cols + col, own[j]);
  }
  auto input = [&](int64_t i, float v[N]) {  // of the sequence's token i, from the state where i < 0
    if (i >= 0) {
      get_some<N>(x + i * args.ld, v);
#pragma unroll
      for (int e = 0; e < N; ++e) v[e] += in_bias[e];
    } else {
#pragma unroll
      for (int e = 0; e < N; ++e) v[e] = 0.f;
      if (held) get_some<N>(state + (back + i) * a.cols, v);
    }
  };
  auto finish = [&](int64_t i, float y[N]) {
#pragma unroll
    for (int e = 0; e < N; ++e)
      if (a.silu) y[e] *= sizeof(Act) == 4 ? sigmoid_f(y[e]) : sigmoid_near(y[e]);
    set_some<N>(static_cast<Act*>(args.out) + (row0 + i) * args.ld_o + col, y);
  };
  if constexpr (TAPS > 0) {
    float past[TAPS][N];  // the inputs of the last TAPS tokens, the current one's last
#pragma unroll
    for (int j = 1; j < TAPS; ++j) input(begin - TAPS + j, past[j]);
    for (int64_t i0 = begin; i0 < end; i0 += CONV_AHEAD) {  // (so many tokens' inputs on their way at once; more, and the loop outgrows the instruction cache)
      float next[CONV_AHEAD][N];
#pragma unroll
      for (int k = 0; k < CONV_AHEAD; ++k)
        if (i0 + k < end) input(i0 + k, next[k]);
#pragma unroll
      for (int k = 0; k < CONV_AHEAD; ++k) {
        if (i0 + k >= end) break;
        float y[N];
#pragma unroll
        for (int e = 0; e < N; ++e) {
#pragma unroll
          for (int j = 0; j + 1 < TAPS; ++j) past[j][e] = past[j + 1][e];
          past[TAPS - 1][e] = next[k][e], y[e] = bias[e];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) y[e] = fmaf(own[j][e], past[j][e], y[e]);
        }
        finish(i0 + k, y);
      }
    }
  } else {
    for (int64_t i = begin; i < end; ++i) {
      float y[N];
#pragma unroll
      for (int e = 0; e < N; ++e) y[e] = bias[e];
      for (int j = 0; j < taps; ++j) {
        float u[N], w[N];
        input(i - back + j, u);
        get_some<N>(a.w + j * a.cols + col, w);
#pragma unroll
        for (int e = 0; e < N; ++e) y[e] = fmaf(w[e], u[e], y[e]);
      }
      finish(i, y);
    }
  }
  if (b == 0 && !dead && back > 0)  // (a thread's own columns, rows rising: what a row is made of is read before it is overwritten)
    for (int r = 0; r < back; ++r) {
      float v[N];
      input(a.tokens + r - back, v);
      set_some<N>(state + r * a.cols, v);
    }
}

template <typename In, typename Act, int N>
static int launch_conv(const ConvArgs& a, cudaStream_t s) {
  const dim3 grid((unsigned)(a.c.sequences * (1 + ceil_div(a.c.tokens - a.first, a.group))), (unsigned)ceil_div(a.c.cols, CONV_THREADS * N)), block(CONV_THREADS);
  switch (a.c.taps) {
    case 2: return launch_after(short_conv_kernel<In, Act, N, 2>, grid, block, 0, s, "fb_short_conv", a);
    case 3: return launch_after(short_conv_kernel<In, Act, N, 3>, grid, block, 0, s, "fb_short_conv", a);
    case CONV_KEPT: return launch_after(short_conv_kernel<In, Act, N, CONV_KEPT>, grid, block, 0, s, "fb_short_conv", a);
    default: return launch_after(short_conv_kernel<In, Act, N, 0>, grid, block, 0, s, "fb_short_conv", a);
  }
}

template <typename In, typename Act>
static int run_conv(ConvArgs a, cudaStream_t s) {
  const fb_conv& c = a.c;
  a.first = (int)(c.taps - 1 < 1 ? 1 : c.taps - 1 < c.tokens ? c.taps - 1 : c.tokens), a.group = CONV_AHEAD;
  while (a.group < 32 && ceil_div(c.sequences * c.tokens, 2 * a.group) * ceil_div(c.cols, CONV_THREADS * 4) >= 32 * 148) a.group *= 2;  // (a run's first token reads the taps - 1 before it)
  auto whole = [](const void* p, int64_t ld, int bytes) { return (uintptr_t)p % (4 * bytes) == 0 && ld % 4 == 0; };
  const bool fours = c.cols % 4 == 0 && whole(a.x, a.ld, sizeof(In)) && whole(a.out, a.ld_o, sizeof(Act)) && whole(c.w, 0, 4) && whole(c.state, c.state_stride, 4);
  return fours ? launch_conv<In, Act, 4>(a, s) : launch_conv<In, Act, 1>(a, s);
}

// ---- the recurrence
struct LruArgs {
  fb_lru l;
  const void* u;
  int64_t ld_u;
  const float* gates;  // [rows, 2 width]: a block's r, then its i
  int64_t ld_gates;
  int part;  // columns of a block
  const void* y;
  int64_t ld_y;
  void* out;
  int64_t ld_o;
};

struct LruColumn {
  float slope, r_bias, i_bias, y_bias;  // slope: log a = slope r
  int64_t r_at;                         // of the gates; i's is `part` on
};

__device__ __forceinline__ LruColumn lru_column(const LruArgs& a, int64_t col) {
  LruColumn c;
  const float lam = a.l.lam[col];
  c.slope = a.l.rate * (fmaxf(lam, 0.f) + log1pf(expf(-fabsf(lam))));
  c.r_at = col / a.part * 2 * a.part + col % a.part;
  c.r_bias = a.l.gate_bias ? a.l.gate_bias[c.r_at] : 0.f, c.i_bias = a.l.gate_bias ? a.l.gate_bias[c.r_at + a.part] : 0.f;
  c.y_bias = a.l.y_bias ? a.l.y_bias[col] : 0.f;
  return c;
}

__device__ __forceinline__ float sqrt_near(float x) {
  float y;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// a token's step: the state becomes a S + b.  1 - a^2 is formed from log a, so that it holds where a is all but 1; NEAR: by the
// hardware's exponential, and there by its power series
template <bool NEAR>
__device__ __forceinline__ void lru_step(const LruColumn& c, float r, float i, float u, float& a, float& b) {
  if constexpr (NEAR) {
    const float log_a = c.slope * sigmoid_near(r + c.r_bias), z = 2.f * log_a;
    a = __expf(log_a);
    const float series = -z * fmaf(z, fmaf(z, fmaf(z, fmaf(z, fmaf(z, 1.f / 720.f, 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
    b = sqrt_near(z > -0.3f ? series : fmaf(-a, a, 1.f)) * sigmoid_near(i + c.i_bias) * u;
  } else {
    const float log_a = c.slope * sigmoid_f(r + c.r_bias);
    a = expf(log_a);
    b = sqrtf(-expm1f(2.f * log_a)) * sigmoid_f(i + c.i_bias) * u;
  }
}

__device__ __forceinline__ float gelu_of(float z) { return 0.5f * z * (1.f + tanh_of(0.7978845608028654f * fmaf(0.044715f * z * z, z, z))); }

template <typename Act, typename Y>
__global__ void __launch_bounds__(128) lru_token_kernel(const LruArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  const int64_t col = (int64_t)blockIdx.x * blockDim.x + threadIdx.x, seq = blockIdx.y;
  if (col >= a.l.width) return;
  const int place = a.l.places[seq];
  Act* out = static_cast<Act*>(a.out) + seq * a.ld_o + col;
  if (place == a.l.dead) return store_value(out, 0.f);
  float* state = a.l.state + seq * a.l.state_stride + col;
  const LruColumn c = lru_column(a, col);
  const float before = *state, r = a.gates[seq * a.ld_gates + c.r_at], i = a.gates[seq * a.ld_gates + c.r_at + a.part];
  const float u = value_of(static_cast<const Act*>(a.u)[seq * a.ld_u + col]), y = value_of(static_cast<const Y*>(a.y)[seq * a.ld_y + col]);
  float decay, in;
  lru_step<sizeof(Act) == 2>(c, r, i, u, decay, in);
  const float s = place ? fmaf(decay, before, in) : in;
  *state = s;
  store_value(out, a.l.scale * s * gelu_of(y + c.y_bias));
}

constexpr int LRU_COLS = 16, LRU_RUNS = 32, LRU_TOKENS = 8;

template <typename Act, typename Y, int BLOCKS>  // BLOCKS: of them an SM (one alone has registers enough to have more on its way)
__global__ void __launch_bounds__(LRU_COLS* LRU_RUNS, BLOCKS) lru_scan_kernel(const LruArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  __shared__ float2 parts[2][LRU_RUNS][LRU_COLS];  // of each run: the product of its a, the state it ends in from zero
  const int lane = threadIdx.x % LRU_COLS, run = threadIdx.x / LRU_COLS;
  const int64_t seq = blockIdx.y, row0 = seq * a.l.tokens, col = (int64_t)blockIdx.x * LRU_COLS + lane;
  const bool mine = col < a.l.width;
  const int place = a.l.places[row0];
  if (place == a.l.dead) {
    for (int64_t t = run; t < a.l.tokens && mine; t += LRU_RUNS) store_value(static_cast<Act*>(a.out) + (row0 + t) * a.ld_o + col, 0.f);
    return;
  }
  const LruColumn c = lru_column(a, mine ? col : 0);
  float* state = a.l.state + seq * a.l.state_stride + col;
  float carry = mine && place ? *state : 0.f;
  const int64_t first = row0 + run * LRU_TOKENS, stride = LRU_RUNS * LRU_TOKENS;
  const Act* u = static_cast<const Act*>(a.u) + first * a.ld_u + col;
  const Y* y = static_cast<const Y*>(a.y) + first * a.ld_y + col;
  const float* gates = a.gates + first * a.ld_gates + c.r_at;
  Act* out = static_cast<Act*>(a.out) + first * a.ld_o + col;
  int buf = 0;
  for (int64_t s0 = 0; s0 < a.l.tokens; s0 += stride, buf ^= 1) {
    float decay[LRU_TOKENS], in[LRU_TOKENS], v[LRU_TOKENS], z[LRU_TOKENS];
    const int n = mine ? (int)min((int64_t)LRU_TOKENS, max((int64_t)0, a.l.tokens - s0 - run * LRU_TOKENS)) : 0;
#pragma unroll
    for (int k = 0; k < LRU_TOKENS; ++k) {  // (all on their way before the first is needed)
      decay[k] = in[k] = v[k] = z[k] = 0.f;
      if (k < n) decay[k] = gates[k * a.ld_gates], in[k] = gates[k * a.ld_gates + a.part], v[k] = value_of(u[k * a.ld_u]), z[k] = value_of(y[k * a.ld_y]);
    }
    float whole = 1.f, end = 0.f;
#pragma unroll
    for (int k = 0; k < LRU_TOKENS; ++k) {
      if (k >= n) break;
      float d, b;
      lru_step<sizeof(Act) == 2>(c, decay[k], in[k], v[k], d, b);
      decay[k] = d, in[k] = b, whole *= d, end = fmaf(d, end, b);
    }
    parts[buf][run][lane] = make_float2(whole, end);
    __syncthreads();
    float s = carry;
#pragma unroll 8
    for (int r = 0; r < LRU_RUNS; ++r) {  // every run's own start, and the segment's end
      if (r == run) s = carry;
      const float2 p = parts[buf][r][lane];
      carry = fmaf(p.x, carry, p.y);
    }
#pragma unroll
    for (int k = 0; k < LRU_TOKENS; ++k) {
      if (k >= n) break;
      s = fmaf(decay[k], s, in[k]);
      store_value(out + k * a.ld_o, a.l.scale * s * gelu_of(z[k] + c.y_bias));
    }
    u += stride * a.ld_u, y += stride * a.ld_y, gates += stride * a.ld_gates, out += stride * a.ld_o;
  }
  if (run == 0 && mine) *state = carry;
}

template <typename Act, typename Y>
static int launch_lru(const LruArgs& a, cudaStream_t s) {
  if (a.l.tokens == 1) return launch_after(lru_token_kernel<Act, Y>, dim3((unsigned)ceil_div(a.l.width, 128), (unsigned)a.l.sequences), dim3(128), 0, s, "fb_lru_scan", a);
  const dim3 grid((unsigned)ceil_div(a.l.width, LRU_COLS), (unsigned)a.l.sequences), block(LRU_COLS * LRU_RUNS);
  if ((int64_t)grid.x * grid.y <= 148) return launch_after(lru_scan_kernel<Act, Y, 1>, grid, block, 0, s, "fb_lru_scan", a);
  return launch_after(lru_scan_kernel<Act, Y, 2>, grid, block, 0, s, "fb_lru_scan", a);
}

}  // namespace fb

extern "C" int fb_short_conv(const fb_conv* conv_host, int in_dtype, const void* x, int64_t ld, int dtype, void* out, int64_t ld_o, void* stream) {
  FB_REQUIRE(conv_host && x && out && conv_host->w && conv_host->places, "fb_short_conv: null pointer");
  const fb_conv& c = *conv_host;
  FB_REQUIRE(c.cols >= 1 && c.taps >= 1 && c.taps <= 4096 && c.sequences >= 1 && c.tokens >= 1 && c.sequences * c.tokens < (1ll << 31), "fb_short_conv: empty, or too many rows or taps");
  FB_REQUIRE(c.taps == 1 || (c.state && (c.sequences == 1 || c.state_stride >= (c.taps - 1) * c.cols)), "fb_short_conv: more than one tap takes a state of taps - 1 rows a sequence");
  FB_REQUIRE(ld >= c.cols && ld_o >= c.cols, "fb_short_conv: row strides too small");
  FB_REQUIRE((in_dtype == FB_BF16 || in_dtype == FB_FP32) && (dtype == FB_BF16 || dtype == FB_FP32) && (in_dtype == FB_FP32 || dtype == FB_BF16),
             "fb_short_conv: bf16 or fp32; fp32 results come from fp32");
  const fb::ConvArgs a{c, x, ld, out, ld_o, 0, 0};
  const auto s = (cudaStream_t)stream;
  if (in_dtype == FB_BF16) return fb::run_conv<uint16_t, uint16_t>(a, s);
  return dtype == FB_BF16 ? fb::run_conv<float, uint16_t>(a, s) : fb::run_conv<float, float>(a, s);
}

extern "C" int fb_lru_scan(const fb_lru* lru_host, int dtype, const void* u, int64_t ld_u, const float* gates, int64_t ld_gates, int y_dtype, const void* y, int64_t ld_y,
                           void* out, int64_t ld_o, void* stream) {
  FB_REQUIRE(lru_host && u && gates && y && out && lru_host->lam && lru_host->places && lru_host->state, "fb_lru_scan: null pointer");
  const fb_lru& l = *lru_host;
  FB_REQUIRE(l.width >= 1 && l.blocks >= 1 && l.width % l.blocks == 0 && l.width < (1ll << 30), "fb_lru_scan: equal blocks of columns (got %lld in %d)", (long long)l.width, l.blocks);
  FB_REQUIRE(l.sequences >= 1 && l.sequences <= 65535 && l.tokens >= 1 && (l.sequences == 1 || l.state_stride >= l.width), "fb_lru_scan: up to 65535 sequences, a state each");
  FB_REQUIRE(ld_u >= l.width && ld_gates >= 2 * l.width && ld_y >= l.width && ld_o >= l.width, "fb_lru_scan: row strides too small");
  FB_REQUIRE((y_dtype == FB_BF16 || y_dtype == FB_FP32) && (dtype == FB_BF16 || dtype == FB_FP32) && (y_dtype == FB_FP32 || dtype == FB_BF16),
             "fb_lru_scan: bf16 or fp32; fp32 results come from fp32");
  const fb::LruArgs a{l, u, ld_u, gates, ld_gates, (int)(l.width / l.blocks), y, ld_y, out, ld_o};
  const auto s = (cudaStream_t)stream;
  if (dtype == FB_FP32) return fb::launch_lru<float, float>(a, s);
  return y_dtype == FB_FP32 ? fb::launch_lru<uint16_t, float>(a, s) : fb::launch_lru<uint16_t, uint16_t>(a, s);
}
