// Linear attention whose state decays: S_t = a_t S_(t-1) + k_t v_t^T (fp32, a [dim, vdim] matrix a head and sequence),
// o_t = S_t^T q_t, and the gated RMSNorm that follows it.
//
//   fb_decay_scan       a fixed decay per head
//   fb_selective_scan   a decay and a step size per head and token (a state space): a_t = exp(-exp(a_log) dt_t), the values times
//                       dt_t, keys and queries shared by groups of heads, and skip times the value beside the output
//   fb_gated_rmsnorm    RMSNorm over the heads' outputs, together or in equal parts, with a gate after or before it
//
// Both scans go token after token - a decode step's one token a sequence, and prompts in fp32 or of odd sizes - or, for bf16
// prompts, in chunks of 64 tokens on tensor-core MMAs (decay_chunk_kernel); longer selective ones in selective_prompt.cu.
#include "launch.cuh"
#include "mma_sync.cuh"
#include "scan.cuh"

namespace fb {

// A CTA keeps 32 columns of one head's state of one sequence in registers: thread (group g, lane) the rows
// 16 g .. 16 g + 15 of column `lane`.  The groups' parts of an output meet in shared memory.
constexpr int SCAN_ROWS = 16;

template <typename Act, bool SELECTIVE>
__global__ void decay_scan_kernel(const ScanArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ float scan_smem[];  // q [dim], k [dim], parts [2][groups][32]
  const int lane = threadIdx.x & 31, g = threadIdx.x >> 5, groups = blockDim.x >> 5;
  const int h = blockIdx.y, col = blockIdx.x * 32 + lane;
  const int64_t seq = blockIdx.z, t0 = seq * a.tokens;
  float *sq = scan_smem, *sk = sq + a.dim, *parts = sk + a.dim;
  const bool mine = col < a.vdim;
  const int place = a.places[t0];
  if (place == a.dead) {
    for (int64_t t = 0; t < a.tokens; ++t)
      if (g == 0 && mine) a.out[(t0 + t) * a.ld_o + (int64_t)h * a.vdim + col] = 0.f;
    return;
  }
  float* state = a.state + seq * a.state_stride + (int64_t)h * a.dim * a.vdim;
  float S[SCAN_ROWS];
#pragma unroll
  for (int i = 0; i < SCAN_ROWS; ++i) {
    const int row = g * SCAN_ROWS + i;
    S[i] = place != 0 && mine && row < a.dim ? state[(int64_t)row * a.vdim + col] : 0.f;
  }
  float decay = 0.f, rate = 0.f, bias = 0.f, skip = 0.f;
  if constexpr (SELECTIVE) rate = -expf(a.a_log[h]), bias = a.step_bias[h], skip = a.skip[h];
  else decay = a.decay[h];
  const int64_t shared_at = (int64_t)(h / a.rep) * a.dim;
  for (int64_t t = 0; t < a.tokens; ++t) {
    const Act* x = static_cast<const Act*>(a.x) + (t0 + t) * a.ld;
    float* part = parts + (t & 1) * groups * 32;
    for (int c = threadIdx.x; c < a.dim; c += blockDim.x) {
      sq[c] = value_of(x[a.q0 + shared_at + c]);
      sk[c] = value_of(x[a.k0 + shared_at + c]);
    }
    float v = mine ? value_of(x[a.v0 + (int64_t)h * a.vdim + col]) : 0.f, beside = 0.f;
    if constexpr (SELECTIVE) {
      const float step = softplus_f(a.step[(t0 + t) * a.ld_step + h] + bias);
      decay = expf(rate * step), beside = skip * v, v *= step;
    }
    __syncthreads();
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < SCAN_ROWS; ++i) {
      const int row = g * SCAN_ROWS + i;
      if (row < a.dim) {
        S[i] = fmaf(decay, S[i], sk[row] * v);
        o = fmaf(S[i], sq[row], o);
      }
    }
    part[g * 32 + lane] = o;
    __syncthreads();
    if (g == 0 && mine) {
      for (int w = 1; w < groups; ++w) o += part[w * 32 + lane];
      a.out[(t0 + t) * a.ld_o + (int64_t)h * a.vdim + col] = o + beside;
    }
  }
#pragma unroll
  for (int i = 0; i < SCAN_ROWS; ++i) {
    const int row = g * SCAN_ROWS + i;
    if (mine && row < a.dim) state[(int64_t)row * a.vdim + col] = S[i];
  }
}

// ---- a prompt in chunks of 64 tokens.  Within a chunk that starts from the state S,
//     o_i = decay^(i+1) S^T q_i + sum over j <= i of decay^(i-j) (q_i . k_j) v_j,    S' = decay^n S + sum decay^(n-1-j) k_j v_j^T,
// all of it matrix products; where the decay is a token's own, decay^(i-j) is the product of those after token j up to token i,
// exp2 of a difference of running sums of their logarithms, and v_j comes times its step.  A CTA walks one sequence's chunks for
// one head and 32 of its value columns, with its part of the state in registers as the accumulators of the last product.  q, k and
// v are bf16 as they come; what is not - the state, the decayed scores, the decayed values - enters a product as two bf16 parts, so
// the recurrence keeps fp32's range and 16 bits of mantissa in every factor, with sums in fp32.
constexpr int CH_TOKENS = 64, CH_COLS = 32, CH_PITCH = CH_COLS * 2 + 16;  // (rows an odd number of 16-byte pieces apart: no bank conflicts)

template <int TILES, bool SELECTIVE>  // TILES: 16-row tiles of the state a warp owns
__global__ void __launch_bounds__(128) decay_chunk_kernel(const ScanArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ __align__(128) uint8_t chunk_smem[];
  __shared__ float power[CH_TOKENS + 1];  // a fixed decay's powers
  __shared__ float2 logs[2][CH_TOKENS];   // selective: log2 of the decays up to and with each token, and its step
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, v0 = blockIdx.x * CH_COLS;
  const int dim = a.dim, pitch = dim * 2 + 16, pieces = dim / 8;
  const int64_t seq = blockIdx.z, t0 = seq * a.tokens;
  const uint32_t sQ = smem_addr(chunk_smem), sK = sQ + 2 * CH_TOKENS * pitch, sV = sK + 2 * CH_TOKENS * pitch;
  const uint32_t sS = sV + 2 * CH_TOKENS * CH_PITCH, sW = sS + 2 * dim * CH_PITCH;  // the state, the decayed values: high parts, then low
  uint8_t* generic = chunk_smem - sQ;  // + a shared address
  const uint16_t* qkv = static_cast<const uint16_t*>(a.x);
  const int64_t q_at = a.q0 + (int64_t)(h / a.rep) * dim, k_at = a.k0 + (int64_t)(h / a.rep) * dim, v_at = a.v0 + (int64_t)h * a.vdim + v0;
  const int place = a.places[t0];
  float rate = 0.f, bias = 0.f, skip = 0.f, raw[2] = {0.f, 0.f};
  if constexpr (SELECTIVE) rate = -expf(a.a_log[h]) * 1.4426950408889634f, bias = a.step_bias[h], skip = a.skip[h];
  else
    for (int e = tid; e <= CH_TOKENS; e += 128) power[e] = (float)pow((double)a.decay[h], (double)e);
  // selective, warp 0: the steps of a chunk's tokens 2 lane and 2 lane + 1 on their way, and, later, what becomes of them
  auto fetch_steps = [&](int64_t c) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int64_t t = c * CH_TOKENS + 2 * lane + e;
      if (t < a.tokens) raw[e] = a.step[(t0 + t) * a.ld_step + h];
    }
  };
  auto put_steps = [&](int64_t c, int buf) {
    float step[2], sum[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) step[e] = c * CH_TOKENS + 2 * lane + e < a.tokens ? softplus_f(raw[e] + bias) : 0.f;  // (past the end: nothing decays, nothing joins)
    sum[0] = rate * step[0], sum[1] = sum[0] + rate * step[1];
    float before = sum[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, before, o);
      if (lane >= o) before += v;
    }
    before -= sum[1];
#pragma unroll
    for (int e = 0; e < 2; ++e) logs[buf][2 * lane + e] = make_float2(before + sum[e], step[e]);
  };

  auto load = [&](int64_t c, int buf) {
    for (int i = tid; i < CH_TOKENS * pieces; i += 128) {
      const int r = i / pieces, ch = i % pieces;
      const int64_t t = c * CH_TOKENS + r;
      const bool in = t < a.tokens;
      const uint16_t* x = qkv + (t0 + (in ? t : 0)) * a.ld + ch * 8;
      cp_async16_or_zero(sQ + (buf * CH_TOKENS + r) * pitch + ch * 16, x + q_at, in ? 16 : 0);
      cp_async16_or_zero(sK + (buf * CH_TOKENS + r) * pitch + ch * 16, x + k_at, in ? 16 : 0);
    }
    for (int i = tid; i < CH_TOKENS * CH_COLS / 8; i += 128) {
      const int r = i / (CH_COLS / 8), ch = i % (CH_COLS / 8);
      const int64_t t = c * CH_TOKENS + r;
      const bool in = t < a.tokens && v0 + ch * 8 < a.vdim;
      cp_async16_or_zero(sV + (buf * CH_TOKENS + r) * CH_PITCH + ch * 16, in ? qkv + (t0 + t) * a.ld + v_at + ch * 8 : qkv, in ? 16 : 0);
    }
    cp_async_commit();
  };
  load(0, 0);
  if (SELECTIVE && warp == 0) fetch_steps(0), put_steps(0, 0);

  float* state = a.state + seq * a.state_stride + (int64_t)h * dim * a.vdim;
  float S[TILES][CH_COLS / 8][4];
  auto each_state = [&](auto&& f) {  // f(value, row, column) for the pairs of this thread's part of the state
#pragma unroll
    for (int i = 0; i < TILES; ++i)
#pragma unroll
      for (int n = 0; n < CH_COLS / 8; ++n)
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          const int row = 16 * (warp + 4 * i) + (lane >> 2) + 8 * g, col = n * 8 + (lane & 3) * 2;
          if (row < dim) f(S[i][n][2 * g], S[i][n][2 * g + 1], row, col);
        }
  };
#pragma unroll
  for (int i = 0; i < TILES; ++i)
#pragma unroll
    for (int n = 0; n < CH_COLS / 8; ++n) S[i][n][0] = S[i][n][1] = S[i][n][2] = S[i][n][3] = 0.f;
  if (place != 0)
    each_state([&](float& x, float& y, int row, int col) {
      if (v0 + col < a.vdim) {  // (vdim is even)
        const float2 v = *reinterpret_cast<const float2*>(state + (int64_t)row * a.vdim + v0 + col);
        x = v.x, y = v.y;
      }
    });

  const int64_t chunks = (a.tokens + CH_TOKENS - 1) / CH_TOKENS;
  const int m = lane >> 3, m_row = lane & 7;
  for (int64_t c = 0; c < chunks; ++c) {
    const int buf = (int)(c & 1), n = (int)min((int64_t)CH_TOKENS, a.tokens - c * CH_TOKENS);
    cp_async_wait<0>();
    __syncthreads();
    if (c + 1 < chunks) load(c + 1, buf ^ 1);
    each_state([&](float& x, float& y, int row, int col) {
      uint32_t high, low;
      split_bf16x2(x, y, high, low);
      *reinterpret_cast<uint32_t*>(generic + sS + row * CH_PITCH + col * 2) = high;
      *reinterpret_cast<uint32_t*>(generic + sS + (dim + row) * CH_PITCH + col * 2) = low;
    });
    for (int i = tid; i < CH_TOKENS * CH_COLS / 2; i += 128) {  // decay^(n-1-j) v_j
      const int j = i / (CH_COLS / 2), at = j * CH_PITCH + (i % (CH_COLS / 2)) * 4;
      const uint32_t v = *reinterpret_cast<const uint32_t*>(generic + sV + buf * CH_TOKENS * CH_PITCH + at);
      float f;
      if constexpr (SELECTIVE) f = exp2_of(logs[buf][CH_TOKENS - 1].x - logs[buf][j].x) * logs[buf][j].y;
      else f = j < n ? power[n - 1 - j] : 0.f;
      uint32_t high, low;
      split_bf16x2(f * bf16_bits_to_float(v & 0xffffu), f * bf16_bits_to_float(v >> 16), high, low);
      *reinterpret_cast<uint32_t*>(generic + sW + at) = high;
      *reinterpret_cast<uint32_t*>(generic + sW + CH_TOKENS * CH_PITCH + at) = low;
    }
    __syncthreads();

    const uint32_t q = sQ + buf * CH_TOKENS * pitch, k = sK + buf * CH_TOKENS * pitch, v = sV + buf * CH_TOKENS * CH_PITCH;
    const int i0 = 16 * warp, row0 = i0 + (lane >> 2);  // this warp's tokens; this thread's are row0 and row0 + 8
    if (SELECTIVE && warp == 0 && c + 1 < chunks) fetch_steps(c + 1);
    if (i0 < n) {
      float o[CH_COLS / 8][4], log_i[2] = {0.f, 0.f}, since[2];  // since: what is left of the state from before the chunk
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        if constexpr (SELECTIVE) log_i[g] = logs[buf][row0 + 8 * g].x, since[g] = exp2_of(log_i[g]);
        else since[g] = power[row0 + 8 * g + 1];
      }
#pragma unroll
      for (int d = 0; d < CH_COLS / 8; ++d) o[d][0] = o[d][1] = o[d][2] = o[d][3] = 0.f;
      for (int kt = 0; kt < dim / 16; ++kt) {  // S^T q
        uint32_t qa[4];
        ldmatrix_x4(q + (i0 + (m & 1) * 8 + m_row) * pitch + (2 * kt + (m >> 1)) * 16, qa);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int d = 0; d < CH_COLS / 8; d += 2) {
            uint32_t b[4];
            ldmatrix_x4_trans(sS + (part * dim + kt * 16 + (m & 1) * 8 + m_row) * CH_PITCH + (d + (m >> 1)) * 16, b);
            mma_bf16(o[d], qa, b[0], b[1]);
            mma_bf16(o[d + 1], qa, b[2], b[3]);
          }
      }
#pragma unroll
      for (int d = 0; d < CH_COLS / 8; ++d) {
        o[d][0] *= since[0], o[d][1] *= since[0];
        o[d][2] *= since[1], o[d][3] *= since[1];
      }
      for (int js = 0; js <= warp; ++js) {  // 16 earlier tokens at a time (the last 16: this warp's own)
        float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        for (int kt = 0; kt < dim / 16; ++kt) {
          uint32_t qa[4], b[4];
          ldmatrix_x4(q + (i0 + (m & 1) * 8 + m_row) * pitch + (2 * kt + (m >> 1)) * 16, qa);
          ldmatrix_x4(k + (16 * js + (m >> 1) * 8 + m_row) * pitch + (2 * kt + (m & 1)) * 16, b);
          mma_bf16(s[0], qa, b[0], b[1]);
          mma_bf16(s[1], qa, b[2], b[3]);
        }
        uint32_t high[4], low[4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int g = 0; g < 2; ++g) {
            const int i = row0 + 8 * g, j = 16 * js + nt * 8 + (lane & 3) * 2;
            float x = 0.f, y = 0.f;
            if constexpr (SELECTIVE) {
              const float2 lx = logs[buf][j], ly = logs[buf][j + 1];
              if (j <= i) x = s[nt][2 * g] * exp2_of(log_i[g] - lx.x) * lx.y;
              if (j + 1 <= i) y = s[nt][2 * g + 1] * exp2_of(log_i[g] - ly.x) * ly.y;
            } else {
              if (j <= i) x = s[nt][2 * g] * power[i - j];
              if (j + 1 <= i) y = s[nt][2 * g + 1] * power[i - j - 1];
            }
            split_bf16x2(x, y, high[2 * nt + g], low[2 * nt + g]);
          }
#pragma unroll
        for (int d = 0; d < CH_COLS / 8; d += 2) {
          uint32_t b[4];
          ldmatrix_x4_trans(v + (16 * js + (m & 1) * 8 + m_row) * CH_PITCH + (d + (m >> 1)) * 16, b);
          mma_bf16(o[d], high, b[0], b[1]);
          mma_bf16(o[d], low, b[0], b[1]);
          mma_bf16(o[d + 1], high, b[2], b[3]);
          mma_bf16(o[d + 1], low, b[2], b[3]);
        }
      }
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        const int i = row0 + 8 * g;
        float* out = a.out + (t0 + c * CH_TOKENS + i) * a.ld_o + (int64_t)h * a.vdim + v0;
#pragma unroll
        for (int d = 0; d < CH_COLS / 8; ++d) {
          const int col = d * 8 + (lane & 3) * 2;
          if (SELECTIVE) {
            const uint32_t own = *reinterpret_cast<const uint32_t*>(generic + v + i * CH_PITCH + col * 2);
            o[d][2 * g] = fmaf(skip, bf16_bits_to_float(own & 0xffffu), o[d][2 * g]), o[d][2 * g + 1] = fmaf(skip, bf16_bits_to_float(own >> 16), o[d][2 * g + 1]);
          }
          if (i < n && v0 + col < a.vdim) *reinterpret_cast<float2*>(out + col) = make_float2(o[d][2 * g], o[d][2 * g + 1]);
        }
      }
    }
    if (SELECTIVE && warp == 0 && c + 1 < chunks) put_steps(c + 1, buf ^ 1);
    // the state after the chunk
    float through;
    if constexpr (SELECTIVE) through = exp2_of(logs[buf][CH_TOKENS - 1].x);
    else through = power[n];
#pragma unroll
    for (int i = 0; i < TILES; ++i) {
      const int tile = warp + 4 * i;
      if (16 * tile >= dim) continue;
#pragma unroll
      for (int d = 0; d < CH_COLS / 8; ++d)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][d][e] *= through;
      for (int js = 0; js < (n + 15) / 16; ++js) {
        uint32_t ka[4];
        ldmatrix_x4_trans(k + (16 * js + (m >> 1) * 8 + m_row) * pitch + (2 * tile + (m & 1)) * 16, ka);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int d = 0; d < CH_COLS / 8; d += 2) {
            uint32_t b[4];
            ldmatrix_x4_trans(sW + (part * CH_TOKENS + 16 * js + (m & 1) * 8 + m_row) * CH_PITCH + (d + (m >> 1)) * 16, b);
            mma_bf16(S[i][d], ka, b[0], b[1]);
            mma_bf16(S[i][d + 1], ka, b[2], b[3]);
          }
      }
    }
  }
  each_state([&](float& x, float& y, int row, int col) {
    if (v0 + col < a.vdim) *reinterpret_cast<float2*>(state + (int64_t)row * a.vdim + v0 + col) = make_float2(x, y);
  });
}

static size_t chunk_smem_bytes(int dim) {
  return 4 * (size_t)CH_TOKENS * (dim * 2 + 16) + 4 * (size_t)CH_TOKENS * CH_PITCH + 2 * (size_t)dim * CH_PITCH;
}

template <int TILES, bool SELECTIVE>
static int launch_chunks(const ScanArgs& a, int64_t sequences, cudaStream_t s) {
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(decay_chunk_kernel<TILES, SELECTIVE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  // (not ahead of the kernel before: long CTAs that find the GPU half full stand two on one SM and none on another)
  decay_chunk_kernel<TILES, SELECTIVE><<<dim3((unsigned)ceil_div(a.vdim, CH_COLS), (unsigned)a.heads, (unsigned)sequences), 128, chunk_smem_bytes(a.dim), s>>>(a);
  return launch_status(SELECTIVE ? "fb_selective_scan (chunks)" : "fb_decay_scan (chunks)");
}

template <bool SELECTIVE>
static int run_scan(int dtype, const ScanArgs& a, int64_t sequences, cudaStream_t s) {
  const char* what = SELECTIVE ? "fb_selective_scan" : "fb_decay_scan";
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "%s: bf16 or fp32", what);
  FB_REQUIRE(a.dim <= 512, "%s: heads of up to 512 query columns (got %d)", what, a.dim);
  FB_REQUIRE(a.ld_o >= (int64_t)a.heads * a.vdim && a.state_stride >= (int64_t)a.heads * a.dim * a.vdim && sequences <= 65535 && a.heads <= 65535, "%s: row strides too small", what);
  if constexpr (SELECTIVE) {
    if (dtype == FB_BF16 && selective_prompt_supports(a, sequences)) return selective_prompt(a, sequences, s);
  }
  // (a few tokens are done sooner one by one)
  if (dtype == FB_BF16 && a.tokens >= 16 && a.dead < 0 && a.dim % 16 == 0 && a.dim <= 256 && a.vdim % 8 == 0 && a.ld % 8 == 0 && a.q0 % 8 == 0 && a.k0 % 8 == 0 && a.v0 % 8 == 0 && a.ld_o % 2 == 0 &&
      a.state_stride % 2 == 0 && (uintptr_t)a.x % 16 == 0 && (uintptr_t)a.state % 8 == 0 && (uintptr_t)a.out % 8 == 0)
    return a.dim <= 64 ? launch_chunks<1, SELECTIVE>(a, sequences, s) : a.dim <= 128 ? launch_chunks<2, SELECTIVE>(a, sequences, s) : launch_chunks<4, SELECTIVE>(a, sequences, s);
  const int groups = (a.dim + SCAN_ROWS - 1) / SCAN_ROWS;
  const dim3 grid((unsigned)ceil_div(a.vdim, 32), (unsigned)a.heads, (unsigned)sequences), block(32 * groups);
  const size_t smem = (2 * (size_t)a.dim + 2 * groups * 32) * sizeof(float);
  if (dtype == FB_FP32) return launch_after(decay_scan_kernel<float, SELECTIVE>, grid, block, smem, s, what, a);
  return launch_after(decay_scan_kernel<uint16_t, SELECTIVE>, grid, block, smem, s, what, a);
}

// V: columns a thread takes at once (4 where rows are aligned); up to NORM_KEPT such pieces a thread stay in registers between the
// sum and the result, a wider row is read again
constexpr int NORM_THREADS = 256, NORM_KEPT = 4;

__device__ __forceinline__ void load4(const float* p, float v[4]) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
}
__device__ __forceinline__ void load4(const uint16_t* p, float v[4]) {
  const uint2 x = *reinterpret_cast<const uint2*>(p);
  v[0] = bf16_bits_to_float(x.x & 0xffffu), v[1] = bf16_bits_to_float(x.x >> 16), v[2] = bf16_bits_to_float(x.y & 0xffffu), v[3] = bf16_bits_to_float(x.y >> 16);
}
__device__ __forceinline__ void store4(float* p, const float v[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(uint16_t* p, const float v[4]) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}
template <int V, typename T>
__device__ __forceinline__ void load_piece(const T* p, float v[V]) {
  if constexpr (V == 4) load4(p, v);
  else v[0] = value_of(*p);
}

// a block a row and part of it.  BEFORE: x times the SiLU of its gate is normed; else the normed x is multiplied by its sigmoid
template <typename Gate, typename Act, int V, bool BEFORE>
__global__ void __launch_bounds__(NORM_THREADS) gated_rmsnorm_kernel(const float* x, int64_t ldx, const void* gate, int64_t ld_g, const float* w, float eps,
                                                                     int64_t cols, void* out, int64_t ldo) {
  griddep_launch_dependents();
  griddep_wait();
  __shared__ float red[32];
  const int64_t t = blockIdx.x, part = blockIdx.y * cols;
  const Gate* g = static_cast<const Gate*>(gate) + t * ld_g + part;
  Act* o = static_cast<Act*>(out) + t * ldo + part;
  x += t * ldx + part, w += part;
  const int64_t c0 = threadIdx.x * V, step = NORM_THREADS * V, kept = NORM_KEPT * step;
  float v[NORM_KEPT][V], f[NORM_KEPT][V], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NORM_KEPT; ++i)
    if (c0 + i * step < cols) load_piece<V>(x + c0 + i * step, v[i]), load_piece<V>(g + c0 + i * step, f[i]);
#pragma unroll
  for (int i = 0; i < NORM_KEPT; ++i)
    if (c0 + i * step < cols) {
      float ws[V];
      load_piece<V>(w + c0 + i * step, ws);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        if (BEFORE) v[i][e] *= f[i][e] * sigmoid_f(f[i][e]), f[i][e] = ws[e];
        else f[i][e] = sigmoid_f(f[i][e]) * ws[e];
        ss = fmaf(v[i][e], v[i][e], ss);
      }
    }
  auto again = [&](int64_t c) { return BEFORE ? x[c] * value_of(g[c]) * sigmoid_f(value_of(g[c])) : x[c]; };
  for (int64_t c = c0 + kept; c < cols; c += step)
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float y = again(c + e);
      ss = fmaf(y, y, ss);
    }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)cols + eps);
#pragma unroll
  for (int i = 0; i < NORM_KEPT; ++i)
    if (c0 + i * step < cols) {
#pragma unroll
      for (int e = 0; e < V; ++e) v[i][e] *= r * f[i][e];
      if constexpr (V == 4) store4(o + c0 + i * step, v[i]);
      else store_value(o + c0 + i * step, v[i][0]);
    }
  for (int64_t c = c0 + kept; c < cols; c += step)
#pragma unroll
    for (int e = 0; e < V; ++e) store_value(o + c + e, again(c + e) * r * w[c + e] * (BEFORE ? 1.f : sigmoid_f(value_of(g[c + e]))));
}

template <typename Gate, typename Act>
static int launch_gated_rmsnorm(const float* x, int64_t rows, int64_t cols, int64_t ldx, const void* gate, int64_t ld_g, bool before, const float* w, float eps, int parts, void* out,
                                int64_t ldo, cudaStream_t s) {
  cols /= parts;
  const bool pieces = cols % 4 == 0 && ldx % 4 == 0 && ld_g % 4 == 0 && ldo % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 &&
                      (uintptr_t)gate % (4 * sizeof(Gate)) == 0 && (uintptr_t)out % (4 * sizeof(Act)) == 0;
  auto kernel = pieces ? before ? gated_rmsnorm_kernel<Gate, Act, 4, true> : gated_rmsnorm_kernel<Gate, Act, 4, false>
                       : before ? gated_rmsnorm_kernel<Gate, Act, 1, true> : gated_rmsnorm_kernel<Gate, Act, 1, false>;
  return launch_after(kernel, dim3((unsigned)rows, (unsigned)parts), dim3(NORM_THREADS), 0, s, "fb_gated_rmsnorm", x, ldx, gate, ld_g, w, eps, cols, out, ldo);
}

}  // namespace fb

extern "C" int fb_decay_scan(int dtype, const void* qkv, int64_t ld, int heads, int dim, int vdim, const float* decay, const int32_t* places, int dead,
                             int64_t sequences, int64_t tokens, float* state, int64_t state_stride, float* out, int64_t ld_o, void* stream) {
  FB_REQUIRE(qkv && decay && places && state && out && sequences >= 1 && tokens >= 1 && heads >= 1 && dim >= 1 && vdim >= 1, "fb_decay_scan: null pointer or empty");
  const int64_t wide = (int64_t)heads * dim;
  FB_REQUIRE(ld >= 2 * wide + (int64_t)heads * vdim, "fb_decay_scan: row strides too small");
  const fb::ScanArgs a{qkv, ld, 0, wide, 2 * wide, 1, heads, dim, vdim, decay, places, dead, tokens, state, state_stride, out, ld_o, nullptr, 0, nullptr, nullptr, nullptr};
  return fb::run_scan<false>(dtype, a, sequences, (cudaStream_t)stream);
}

extern "C" int fb_selective_scan(int dtype, const void* xbc, int64_t ld, int heads, int groups, int dim, int vdim, const float* step, int64_t ld_step, const float* step_bias,
                                 const float* a_log, const float* skip, const int32_t* places, int dead, int64_t sequences, int64_t tokens, float* state, int64_t state_stride,
                                 float* out, int64_t ld_o, void* stream) {
  FB_REQUIRE(xbc && step && step_bias && a_log && skip && places && state && out && sequences >= 1 && tokens >= 1 && dim >= 1 && vdim >= 1, "fb_selective_scan: null pointer or empty");
  FB_REQUIRE(heads >= 1 && groups >= 1 && heads % groups == 0, "fb_selective_scan: whole groups of heads (got %d / %d)", heads, groups);
  const int64_t inner = (int64_t)heads * vdim, wide = (int64_t)groups * dim;
  FB_REQUIRE(ld >= inner + 2 * wide && ld_step >= heads, "fb_selective_scan: row strides too small");
  const fb::ScanArgs a{xbc, ld, inner + wide, inner, 0, heads / groups, heads, dim, vdim, nullptr, places, dead, tokens, state, state_stride, out, ld_o, step, ld_step, step_bias, a_log, skip};
  return fb::run_scan<true>(dtype, a, sequences, (cudaStream_t)stream);
}

extern "C" int fb_gated_rmsnorm(const float* x, int64_t rows, int64_t cols, int64_t ldx, int gate_dtype, const void* gate, int64_t ld_g, int before, const float* w, float eps, int parts,
                                int dtype, void* out, int64_t ldo, void* stream) {
  FB_REQUIRE(x && gate && w && out && rows >= 1 && cols >= 1 && ldx >= cols && ld_g >= cols && ldo >= cols, "fb_gated_rmsnorm: bad arguments");
  FB_REQUIRE(parts >= 1 && parts <= 65535 && cols % parts == 0, "fb_gated_rmsnorm: equal parts of a row (got %lld columns in %d)", (long long)cols, parts);
  FB_REQUIRE((gate_dtype == FB_BF16 || gate_dtype == FB_FP32) && (dtype == FB_BF16 || dtype == FB_FP32) && (gate_dtype == FB_FP32 || dtype == FB_BF16),
             "fb_gated_rmsnorm: bf16 or fp32; fp32 results take fp32 gates");
  const auto s = (cudaStream_t)stream;
  if (gate_dtype == FB_BF16) return fb::launch_gated_rmsnorm<uint16_t, uint16_t>(x, rows, cols, ldx, gate, ld_g, before, w, eps, parts, out, ldo, s);
  if (dtype == FB_BF16) return fb::launch_gated_rmsnorm<float, uint16_t>(x, rows, cols, ldx, gate, ld_g, before, w, eps, parts, out, ldo, s);
  return fb::launch_gated_rmsnorm<float, float>(x, rows, cols, ldx, gate, ld_g, before, w, eps, parts, out, ldo, s);
}
