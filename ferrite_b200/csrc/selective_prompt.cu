// A prompt of fb_selective_scan on the 5th-generation tensor cores (bf16 rows): the state space in chunks of 128 tokens.
//
// With l_i the running sum of the log decays up to and with token i of a chunk, q, k, x its rows, d its step sizes and S the state
// before it,
//
//   out_i = exp(l_i) S^T q_i + sum over j <= i of exp(l_i - l_j) d_j (q_i . k_j) x_j + skip x_i,
//   S'    = exp(l_last) S + sum over j of k_j (exp(l_last - l_j) d_j x_j)^T.
//
// A CTA walks one sequence's chunks for one head and up to 64 of its value columns; per chunk, accumulators in tensor memory:
//
//   G  [128 tokens, 128 tokens]  = Q . K^T           both K-major, as they lie
//   Y1 [128 tokens, columns]     = Q . S             S the MN-major operand, written by threads
//   Y2 [128 tokens, columns]     = P . X             P = G times decays and steps, from tensor memory; X as it lies, MN-major
//   D  [state rows, columns]     = K^T . W           both MN-major: K as it lies, W = X times decays to the chunk's end and steps
//
// Q, K and X are bf16 as they come; S, P and W enter as two bf16 parts each, so every factor of the recurrence keeps 16 bits of
// mantissa, and sums are fp32.  The state itself stays in fp32 registers from chunk to chunk.
//
//   warps 0-3, 4-7   P of a chunk's first and second 64 keys; the results, 32 columns each
//   warps 8-11, 12-15  W and the state, a row a thread, 32 columns each
//   warp 16  TMA      warp 17  MMAs      warp 18  steps and log decays
//
// The next chunk's G is computed while this one's P is.  Every wait is bounded (sm100.cuh).
#include "mma_sync.cuh"
#include "scan.cuh"
#include "sm100.cuh"
#include "tma_host.cuh"

namespace fb {

namespace {

constexpr int SP_TOKENS = 128, SP_COLS = 64, SP_SLOTS = 4;
constexpr int SP_CHUNK = SP_TOKENS * 128, SP_SLOT = 2 * SP_CHUNK;  // 64 columns of a chunk's rows; a chunk's queries or keys
constexpr int SP_X = SP_SLOTS * SP_SLOT, SP_W = SP_X + 2 * SP_CHUNK, SP_S = SP_W + 2 * SP_CHUNK, SP_SMEM = SP_S + 2 * SP_CHUNK + 1024;
constexpr int SP_Y1 = 2 * SP_TOKENS, SP_Y2 = SP_Y1 + SP_COLS, SP_D = SP_Y2 + SP_COLS, SP_TMEM = 512;
constexpr int PIECE = 16;  // keys of P at a time
constexpr int SP_WARP_LOAD = 16, SP_WARP_MMA = 17, SP_WARP_STEPS = 18, SP_THREADS = 19 * 32;

enum ScanWait { SW_SLOT_EMPTY = 701, SW_SLOT_FULL, SW_X_EMPTY, SW_X_FULL, SW_G, SW_P, SW_Y, SW_Y_EMPTY, SW_W, SW_D, SW_S, SW_Y1, SW_L, SW_L_EMPTY, SW_DRAIN };

// eight values as two bf16 parts, to the swizzled place of their 16 bytes in a row of 128
__device__ __forceinline__ void put_parts(uint32_t row_addr, int unit, int row, const float v[8]) {
  uint32_t high[4], low[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) split_bf16x2(v[2 * e], v[2 * e + 1], high[e], low[e]);
  const uint32_t at = row_addr + ((unit ^ (row & 7)) << 4);
  st_shared_v4(at, high[0], high[1], high[2], high[3]);
  st_shared_v4(at + SP_CHUNK, low[0], low[1], low[2], low[3]);
}
__device__ __forceinline__ uint4 get_eight(const uint8_t* row, int unit, int r) { return *reinterpret_cast<const uint4*>(row + ((unit ^ (r & 7)) << 4)); }
__device__ __forceinline__ void widen(const uint4& x, float v[8]) {
  const uint32_t w[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) v[2 * e] = bf16_bits_to_float(w[e] & 0xffffu), v[2 * e + 1] = bf16_bits_to_float(w[e] >> 16);
}

__global__ void __launch_bounds__(SP_THREADS, 1) selective_prompt_kernel(const __grid_constant__ CUtensorMap map, const ScanArgs a) {
  extern __shared__ uint8_t scan_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(scan_smem) + 1023) & ~uintptr_t(1023));
  __shared__ float2 logs[SP_TOKENS];  // log2: of the decays up to and with a token, and that less its step's
  __shared__ uint64_t bars[2 * SP_SLOTS + 4 + 2 + 2 + 8];
  __shared__ uint32_t tmem_slot[2];  // the allocation's address, the abort flag
  uint64_t *slot_full = bars, *slot_empty = bars + SP_SLOTS, *x_full = bars + 2 * SP_SLOTS, *x_empty = x_full + 2, *g_full = x_empty + 2, *p_full = g_full + 2, *y_full = p_full + 2;
  uint64_t *y_empty = y_full + 1, *y1_done = y_full + 2, *w_full = y_full + 3, *d_full = y_full + 4, *s_full = y_full + 5, *l_full = y_full + 6, *l_empty = y_full + 7;
  const uint32_t abort_flag = smem_u32(tmem_slot + 1);
  const int tid = threadIdx.x, warp = uniform_warp(), lane = tid & 31, h = blockIdx.y, v0 = blockIdx.x * SP_COLS;
  const int cols = min(SP_COLS, a.vdim - v0), wide = (cols + 15) / 16 * 16, n = (int)((a.tokens + SP_TOKENS - 1) / SP_TOKENS);
  const int64_t row0 = blockIdx.z * a.tokens;

  griddep_launch_dependents();
  if (tid == 0) {
    for (int i = 0; i < SP_SLOTS; ++i) mbar_init(smem_u32(slot_full + i), 1), mbar_init(smem_u32(slot_empty + i), 1);
    for (int i = 0; i < 2; ++i) mbar_init(smem_u32(x_full + i), 1), mbar_init(smem_u32(x_empty + i), 17), mbar_init(smem_u32(g_full + i), 1), mbar_init(smem_u32(p_full + i), 8);
    mbar_init(smem_u32(y_full), 1), mbar_init(smem_u32(y_empty), 8), mbar_init(smem_u32(y1_done), 1), mbar_init(smem_u32(w_full), 8);
    mbar_init(smem_u32(d_full), 1), mbar_init(smem_u32(s_full), 8), mbar_init(smem_u32(l_full), 1), mbar_init(smem_u32(l_empty), 16);
    tmem_slot[1] = 0;
    fence_barrier_init();
  }
  if (warp == SP_WARP_MMA) tmem_alloc(smem_u32(tmem_slot), SP_TMEM);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot[0], base = smem_u32(smem), lanes = (uint32_t)(32 * (warp & 3)) << 16;
  const int row = 32 * (warp & 3) + lane;  // of the first sixteen warps: a token of the chunk, or a row of the state
  griddep_wait();

  if (warp == SP_WARP_LOAD && lane == 0) {
    prefetch_tensormap(&map);
    const int pieces = (a.dim + 63) / 64, group = h / a.rep;
    const int at[2] = {(int)(a.q0 + (int64_t)group * a.dim), (int)(a.k0 + (int64_t)group * a.dim)};
    int i = 0;
    bool ok = true;
    for (int c = 0; c < n && ok; ++c) {
      const int y = (int)row0 + c * SP_TOKENS;
      for (int what = 0; what < 2; ++what, ++i) {  // queries, then keys
        const int slot = i % SP_SLOTS;
        ok = mbar_wait(smem_u32(slot_empty + slot), ((i / SP_SLOTS) & 1) ^ 1, abort_flag, SW_SLOT_EMPTY);
        if (!ok) break;
        mbar_expect_tx(smem_u32(slot_full + slot), (uint32_t)pieces * SP_CHUNK);
        for (int p = 0; p < pieces; ++p) tma_load_2d(base + slot * SP_SLOT + p * SP_CHUNK, &map, at[what] + 64 * p, y, smem_u32(slot_full + slot));
      }
      if (!ok) break;
      ok = mbar_wait(smem_u32(x_empty + (c & 1)), ((c >> 1) & 1) ^ 1, abort_flag, SW_X_EMPTY);
      if (!ok) break;
      mbar_expect_tx(smem_u32(x_full + (c & 1)), SP_CHUNK);
      tma_load_2d(base + SP_X + (c & 1) * SP_CHUNK, &map, (int)(a.v0 + (int64_t)h * a.vdim) + v0, y, smem_u32(x_full + (c & 1)));
    }
    if (!ok) {  // given up: the copies under way land before this CTA's shared memory is anyone else's
      const long long start = clock64();
      for (int b = i - 1; b >= 0 && b >= i - SP_SLOTS; --b)
        while (!mbar_try_wait(smem_u32(slot_full + b % SP_SLOTS), (b / SP_SLOTS) & 1) && clock64() - start < WAIT_CLOCKS) {
        }
      for (int c = i / 2 - 1; c >= 0 && c >= i / 2 - 2; --c)
        while (!mbar_try_wait(smem_u32(x_full + (c & 1)), (c >> 1) & 1) && clock64() - start < WAIT_CLOCKS) {
        }
    }
  } else if (warp == SP_WARP_MMA) {
    const uint32_t idesc_g = umma_idesc_bf16(SP_TOKENS, false, false), idesc_y = umma_idesc_bf16(wide, false, true), idesc_d = umma_idesc_bf16(wide, true, true);
    const uint64_t plain0 = umma_smem_desc(base, 16, 1024), turned0 = umma_smem_desc(base, SP_CHUNK, 1024);  // of slot 0, K-major and MN-major
    const uint64_t dx0 = umma_smem_desc(base + SP_X, SP_CHUNK, 1024), dw = umma_smem_desc(base + SP_W, SP_CHUNK, 1024), ds = umma_smem_desc(base + SP_S, SP_CHUNK, 1024);
    constexpr uint32_t slot_step = SP_SLOT >> 4, chunk_step = SP_CHUNK >> 4, rows16 = 2048 >> 4;
    const int nk = a.dim / 16;
    auto scores = [&](int c) {
      const int q = 2 * c % SP_SLOTS, k = (2 * c + 1) % SP_SLOTS;
      mbar_wait(smem_u32(slot_full + q), (2 * c / SP_SLOTS) & 1, abort_flag, SW_SLOT_FULL);
      mbar_wait(smem_u32(slot_full + k), ((2 * c + 1) / SP_SLOTS) & 1, abort_flag, SW_SLOT_FULL);
      tc_fence_after();
#pragma unroll 1
      for (int j = 0; j < nk; ++j) {
        const uint32_t at = (j >> 2) * chunk_step + 2 * (j & 3);
        umma_bf16_warp(tmem + (c & 1) * SP_TOKENS, plain0 + q * slot_step + at, plain0 + k * slot_step + at, idesc_g, j);
      }
      umma_commit_warp(smem_u32(g_full + (c & 1)));
    };
    // (loops that stay in the instruction cache: written out, an MMA waits for its instructions)
    scores(0);
    for (int c = 0; c < n; ++c) {
      const int q = 2 * c % SP_SLOTS, k = (2 * c + 1) % SP_SLOTS;
      if (c + 1 < n) {  // over the P of the chunk before this one, once that is used up
        if (c > 0) mbar_wait(smem_u32(y_full), (c - 1) & 1, abort_flag, SW_Y);
        scores(c + 1);
      }
      // Q . S, once the state is there and the results before are read
      mbar_wait(smem_u32(s_full), c & 1, abort_flag, SW_S);
      if (c > 0) mbar_wait(smem_u32(y_empty), (c - 1) & 1, abort_flag, SW_Y_EMPTY);
      tc_fence_after();
#pragma unroll 1
      for (int j = 0; j < nk; ++j)
#pragma unroll
        for (int part = 0; part < 2; ++part)
          umma_bf16_warp(tmem + SP_Y1, plain0 + q * slot_step + (j >> 2) * chunk_step + 2 * (j & 3), ds + part * chunk_step + j * rows16, idesc_y, part | j);
      umma_commit_warp(smem_u32(slot_empty + q));  // (its scores are done, too)
      umma_commit_warp(smem_u32(y1_done));
      // K^T . W
      mbar_wait(smem_u32(w_full), c & 1, abort_flag, SW_W);
      tc_fence_after();
#pragma unroll 1
      for (int j = 0; j < SP_TOKENS / 16; ++j)
#pragma unroll
        for (int part = 0; part < 2; ++part) umma_bf16_warp(tmem + SP_D, turned0 + k * slot_step + j * rows16, dw + part * chunk_step + j * rows16, idesc_d, part | j);
      umma_commit_warp(smem_u32(slot_empty + k));
      umma_commit_warp(smem_u32(d_full));
      // P . X: of each 16 keys the high parts of P are 8 columns, then the low parts
      mbar_wait(smem_u32(p_full + (c & 1)), (c >> 1) & 1, abort_flag, SW_P);
      mbar_wait(smem_u32(x_full + (c & 1)), (c >> 1) & 1, abort_flag, SW_X_FULL);
      tc_fence_after();
#pragma unroll 1
      for (int j = 0; j < SP_TOKENS / 16; ++j)
#pragma unroll
        for (int part = 0; part < 2; ++part)
          umma_bf16_ts_warp(tmem + SP_Y2, tmem + (c & 1) * SP_TOKENS + j * 16 + part * 8, dx0 + (c & 1) * chunk_step + j * rows16, idesc_y, part | j);
      umma_commit_warp(smem_u32(x_empty + (c & 1)));
      umma_commit_warp(smem_u32(y_full));
    }
  } else if (warp == SP_WARP_STEPS) {
    const float rate = -expf(a.a_log[h]) * 1.4426950408889634f, bias = a.step_bias[h];
    float raw[4] = {0.f, 0.f, 0.f, 0.f};
    auto fetch = [&](int c) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int64_t t = (int64_t)c * SP_TOKENS + 4 * lane + e;
        if (t < a.tokens) raw[e] = a.step[(row0 + t) * a.ld_step + h];
      }
    };
    fetch(0);
    for (int c = 0; c < n; ++c) {
      float step[4], sum[4], total = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {  // (past the end: nothing decays, nothing joins)
        step[e] = (int64_t)c * SP_TOKENS + 4 * lane + e < a.tokens ? softplus_f(raw[e] + bias) : 0.f;
        sum[e] = total += rate * step[e];
      }
      if (c + 1 < n) fetch(c + 1);
      float before = total;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, before, o);
        if (lane >= o) before += v;
      }
      before -= total;
      if (c > 0) mbar_wait(smem_u32(l_empty), (c - 1) & 1, abort_flag, SW_L_EMPTY);
#pragma unroll
      for (int e = 0; e < 4; ++e) logs[4 * lane + e] = make_float2(before + sum[e], before + sum[e] - log2f(step[e]));
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(l_full));
    }
  } else if (warp < 8) {
    const int half = warp >> 2;
    const float skip = a.skip[h];
    // G to P; returns what is left at this token of the state from before the chunk
    auto weigh = [&](int c) {
      mbar_wait(smem_u32(l_full), c & 1, abort_flag, SW_L);
      mbar_wait(smem_u32(g_full + (c & 1)), (c >> 1) & 1, abort_flag, SW_G);
      tc_fence_after();
      const uint32_t at = tmem + lanes + (c & 1) * SP_TOKENS + 64 * half;
      const float mine = logs[row].x;
      // (a loop that stays in the instruction cache: written out in full it waits for its instructions)
#pragma unroll 1
      for (int b = 0; b < 64; b += PIECE) {
        float s[PIECE], parts[PIECE];
        const int key0 = 64 * half + b;
        if (key0 > 32 * (warp & 3) + 31) {  // (keys past all of the warp's tokens)
#pragma unroll
          for (int j = 0; j < PIECE; ++j) parts[j] = 0.f;
        } else {
#pragma unroll
          for (int i = 0; i < PIECE; i += 16) tmem_ld16_nowait(at + b + i, s + i);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < PIECE; j += 2) {
            const int key = key0 + j;
            const float4 l = *reinterpret_cast<const float4*>(logs + key);
            // (of what a token does not see 2^-inf: a choice of the exponent, not a branch)
            uint32_t high, low;
            split_bf16x2(s[j] * exp2_of(key <= row ? mine - l.y : -INFINITY), s[j + 1] * exp2_of(key + 1 <= row ? mine - l.w : -INFINITY), high, low);
            parts[j / 16 * 16 + j % 16 / 2] = __uint_as_float(high), parts[j / 16 * 16 + 8 + j % 16 / 2] = __uint_as_float(low);
          }
        }
#pragma unroll
        for (int i = 0; i < PIECE; i += 16) tmem_st16(at + b + i, parts + i);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(p_full + (c & 1))), mbar_arrive(smem_u32(l_empty));
      return exp2_of(mine);
    };
    float since = 0.f, next = weigh(0);
    for (int c = 0; c < n; ++c) {
      since = next;
      if (c + 1 < n) next = weigh(c + 1);
      mbar_wait(smem_u32(y_full), c & 1, abort_flag, SW_Y);
      tc_fence_after();
      float y[32], z[32];
      tmem_ld32_nowait(tmem + lanes + SP_Y1 + 32 * half, y);
      tmem_ld32_nowait(tmem + lanes + SP_Y2 + 32 * half, z);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(y_empty));
      mbar_wait(smem_u32(x_full + (c & 1)), (c >> 1) & 1, abort_flag, SW_X_FULL);
      const uint8_t* x = smem + SP_X + (c & 1) * SP_CHUNK + row * 128;
      const int64_t t = (int64_t)c * SP_TOKENS + row;
      float* out = a.out + (row0 + t) * a.ld_o + (int64_t)h * a.vdim + v0;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int unit = 4 * half + u;
        float v[8];
        widen(get_eight(x, unit, row), v);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = fmaf(skip, v[e], fmaf(since, y[8 * u + e], z[8 * u + e]));
        if (t < a.tokens && 8 * unit < cols) {
          *reinterpret_cast<float4*>(out + 8 * unit) = make_float4(v[0], v[1], v[2], v[3]);
          *reinterpret_cast<float4*>(out + 8 * unit + 4) = make_float4(v[4], v[5], v[6], v[7]);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(x_empty + (c & 1)));
    }
  } else if (warp < 16) {
    const int first = 32 * (warp >> 2 & 1);  // its columns
    float* state = a.state + blockIdx.z * a.state_stride + ((int64_t)h * a.dim + row) * a.vdim + v0 + first;
    const bool mine = row < a.dim;
    const bool begun = a.places[row0] != 0;
    float S[32];
#pragma unroll
    for (int c = 0; c < 32; c += 4) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (mine && begun && first + c < cols) v = *reinterpret_cast<const float4*>(state + c);
      S[c] = v.x, S[c + 1] = v.y, S[c + 2] = v.z, S[c + 3] = v.w;
    }
    auto put_state = [&] {
      if (mine)
#pragma unroll
        for (int u = 0; u < 4; ++u) put_parts(base + SP_S + row * 128, first / 8 + u, row, S + 8 * u);
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(s_full));
    };
    put_state();
    for (int c = 0; c < n; ++c) {
      mbar_wait(smem_u32(l_full), c & 1, abort_flag, SW_L);
      mbar_wait(smem_u32(x_full + (c & 1)), (c >> 1) & 1, abort_flag, SW_X_FULL);
      const float last = logs[SP_TOKENS - 1].x, f = exp2_of(last - logs[row].y), through = exp2_of(last);
      const uint8_t* x = smem + SP_X + (c & 1) * SP_CHUNK + row * 128;
#pragma unroll 1
      for (int u = first / 8; u < first / 8 + 4; ++u) {
        float v[8];
        widen(get_eight(x, u, row), v);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= f;
        put_parts(base + SP_W + row * 128, u, row, v);
      }
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(w_full)), mbar_arrive(smem_u32(x_empty + (c & 1))), mbar_arrive(smem_u32(l_empty));
      mbar_wait(smem_u32(d_full), c & 1, abort_flag, SW_D);
      tc_fence_after();
#pragma unroll
      for (int b = 0; b < 32; b += 16) {
        float v[16];
        tmem_ld16_nowait(tmem + lanes + SP_D + first + b, v);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 16; ++e) S[b + e] = fmaf(through, S[b + e], v[e]);
      }
      tc_fence_before();
      if (c + 1 < n) {
        mbar_wait(smem_u32(y1_done), c & 1, abort_flag, SW_Y1);
        put_state();
      }
    }
    if (mine)
#pragma unroll
      for (int c = 0; c < 32; c += 4)
        if (first + c < cols) *reinterpret_cast<float4*>(state + c) = make_float4(S[c], S[c + 1], S[c + 2], S[c + 3]);
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (warp == SP_WARP_MMA) {
    tc_fence_after();
    tmem_dealloc(tmem, SP_TMEM);
  }
}

}  // namespace

static const StatusWord g_status_reader(read_and_clear_status_word);

// rows that TMA takes, states of up to 128 rows, more tokens than the chunks of 64 do sooner
bool selective_prompt_supports(const ScanArgs& a, int64_t sequences) {
  return a.tokens > 64 && a.dead < 0 && a.dim % 16 == 0 && a.dim <= 128 && a.vdim % 8 == 0 && a.ld % 8 == 0 && a.q0 % 8 == 0 && a.k0 % 8 == 0 && a.v0 % 8 == 0 && a.ld_o % 4 == 0 &&
         a.state_stride % 4 == 0 && (uintptr_t)a.x % 16 == 0 && (uintptr_t)a.state % 16 == 0 && (uintptr_t)a.out % 16 == 0 && sequences * a.tokens < (1ll << 31) && a.ld < (1ll << 31) &&
         tma_encoder() != nullptr;
}

int selective_prompt(const ScanArgs& a, int64_t sequences, cudaStream_t s) {
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(selective_prompt_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SP_SMEM);
  CUtensorMap map;
  const int64_t groups = a.heads / a.rep, dims[2] = {(int64_t)a.heads * a.vdim + 2 * groups * a.dim, sequences * a.tokens}, strides[1] = {a.ld};
  const int box[2] = {64, SP_TOKENS};
  if (int rc = tma_map_bf16(&map, a.x, 2, dims, strides, box, "fb_selective_scan (rows)")) return rc;
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3((unsigned)ceil_div(a.vdim, SP_COLS), (unsigned)a.heads, (unsigned)sequences), cfg.blockDim = dim3(SP_THREADS);
  cfg.dynamicSmemBytes = SP_SMEM, cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr, cfg.numAttrs = 1;
  cudaLaunchKernelEx(&cfg, selective_prompt_kernel, map, a);
  return launch_status("fb_selective_scan");
}

}  // namespace fb
