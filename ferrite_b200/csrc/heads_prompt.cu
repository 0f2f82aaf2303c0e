// A prompt's chunk of fb_heads_attention on the 5th-generation tensor cores (bf16 rows).
//
// A CTA has one key head and one or two groups of up to 128 (token, query head) pairs - whole tokens, the query heads that
// share the key head side by side, so the rows of a group are one TMA box of q - and walks the keys that its tokens see in
// tiles of 64, each brought in once for both groups:
//
//   scores   S [128 pairs, 64 keys]      = Q . K^T    both from shared memory, K-major
//   sums     O [128 pairs, value columns] += P . V    P from tensor memory, V (as it lies: keys by columns) the MN-major operand
//
// A softmax thread owns a pair: its scores, its probabilities (written over the scores, as bf16) and its sums are one lane of
// tensor memory.  The sums stand under a reference maximum that moves only when the scores outgrow it by a factor of 256.
// Where weights are sigmoids (SIGMOID) there is neither a maximum nor a denominator.
//
//   warps 0-3, 4-7   softmax of the two groups       warp 8   TMA        warp 9   MMAs (the whole warp issues them, written out)
//
// A group's scores alternate between two buffers: the next tile's are computed while this one's softmax runs; the other group's
// MMAs fill the rest.  Every wait is bounded (sm100.cuh).
#include "heads.cuh"
#include "sm100.cuh"
#include "tma_host.cuh"

namespace fb {

namespace {

constexpr int HP_KEYS = 64, HP_MAX_STAGES = 6, HP_ROWS = 128;
constexpr size_t HP_SMEM = 224 * 1024, HP_SMEM_HALF = 112 * 1024;  // a CTA's alone on its SM, one of two
constexpr int HP_Q_CHUNK = HP_ROWS * 128, HP_K_CHUNK = HP_KEYS * 128;  // 64 columns of a group's queries, of a tile's keys or values
constexpr int HP_COLS = 2 * HP_KEYS + 128;                             // tensor memory of a group (of two): two tiles of scores, the sums
constexpr float HP_SLACK = 8.f;                                        // log2 of how far scores may outgrow the reference maximum
constexpr float HP_LOG2E = 1.4426950408889634f;

enum PromptWait { PW_Q = 501, PW_EMPTY, PW_FULL, PW_S, PW_P, PW_PV, PW_PV_MMA, PW_DRAIN };

struct PromptParams {
  HeadsArgs a;
  int groups, tokens;  // tokens of a group
  int fours;           // gates and results are whole, aligned groups of four columns
  int ck, cv, nv, stages, q_bytes, tmem_cols, smem;  // 64-column pieces of a query / key and of a value; columns of the sums; bytes from one group's queries to the next's
};

// v times the sigmoid of g
__device__ __forceinline__ float gated(float v, float g) { return __fdividef(v, 1.f + __expf(-g)); }

template <int GROUPS, bool SIGMOID>
__global__ void __launch_bounds__((4 * GROUPS + 2) * 32, GROUPS == 1 ? 2 : 1) heads_prompt_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tkv, const PromptParams p) {
  constexpr int HP_WARP_LOAD = 4 * GROUPS, HP_WARP_MMA = HP_WARP_LOAD + 1;
  extern __shared__ uint8_t prompt_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(prompt_smem) + 1023) & ~uintptr_t(1023));
  __shared__ uint64_t bars[2 * HP_MAX_STAGES + 10];
  __shared__ uint32_t tmem_slot[2];  // the allocation's address, the abort flag
  uint64_t *full = bars, *empty = bars + HP_MAX_STAGES, *q_full = bars + 2 * HP_MAX_STAGES, *s_full = q_full + 2, *p_full = s_full + 4, *pv_done = p_full + 2;
  const uint32_t abort_flag = smem_u32(tmem_slot + 1);
  const HeadsArgs& a = p.a;
  const int tid = threadIdx.x, warp = uniform_warp(), lane = tid & 31, g = blockIdx.x, S = p.stages;
  const int tile = gridDim.y - 1 - blockIdx.y;  // (the last see the most keys: they start first)
  const uint32_t sQ = smem_u32(smem), sKV = sQ + GROUPS * p.q_bytes, stage_bytes = (p.ck + p.cv) * HP_K_CHUNK;

  griddep_launch_dependents();
  if (tid == 0) {
    for (int i = 0; i < S; ++i) mbar_init(smem_u32(full + i), 1), mbar_init(smem_u32(empty + i), 1);
    for (int i = 0; i < 2; ++i) mbar_init(smem_u32(q_full + i), 1), mbar_init(smem_u32(p_full + i), 4), mbar_init(smem_u32(pv_done + i), 1);
    for (int i = 0; i < 4; ++i) mbar_init(smem_u32(s_full + i), 1);
    tmem_slot[1] = 0;
    fence_barrier_init();
  }
  if (warp == HP_WARP_MMA) tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot[0];
  griddep_wait();

  // the keys that the CTA's tokens see
  const int t0 = tile * GROUPS * p.tokens, t1 = min((int)a.T, t0 + GROUPS * p.tokens);
  int len = 0, lo = 0x7fffffff;
  for (int t = t0 + lane; t < t1; t += 32) {
    const int at = a.last[t];
    len = max(len, at + 1), lo = min(lo, first_seen(a, at));
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) len = max(len, __shfl_xor_sync(0xffffffffu, len, o)), lo = min(lo, __shfl_xor_sync(0xffffffffu, lo, o));
  len = (int)max((int64_t)0, min((int64_t)len, a.cache_rows - a.row0));
  const int k0 = max(0, min(lo, len)), n_tiles = (len - k0 + HP_KEYS - 1) / HP_KEYS;

  if (warp == HP_WARP_LOAD && lane == 0) {
    prefetch_tensormap(&tq), prefetch_tensormap(&tkv);
    if (n_tiles)
      for (int gr = 0; gr < GROUPS; ++gr) {
        mbar_expect_tx(smem_u32(q_full + gr), (uint32_t)(p.ck * p.tokens * a.rep * 128));
        for (int c = 0; c < p.ck; ++c) tma_load_4d(sQ + gr * p.q_bytes + c * HP_Q_CHUNK, &tq, 64 * c, 0, g, t0 + gr * p.tokens, smem_u32(q_full + gr));
      }
    int slot = 0, i = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (; i < n_tiles; ++i) {
      ok = mbar_wait(smem_u32(empty + slot), phase ^ 1, abort_flag, PW_EMPTY);
      if (!ok) break;
      mbar_expect_tx(smem_u32(full + slot), stage_bytes);
      const int row = (int)a.row0 + k0 + i * HP_KEYS;
      const uint32_t to = sKV + slot * stage_bytes;
      for (int c = 0; c < p.ck; ++c) tma_load_3d(to + c * HP_K_CHUNK, &tkv, 64 * c, row, g, smem_u32(full + slot));
      for (int c = 0; c < p.cv; ++c) tma_load_3d(to + (p.ck + c) * HP_K_CHUNK, &tkv, a.dim + 64 * c, row, g, smem_u32(full + slot));
      if (++slot == S) slot = 0, phase ^= 1;
    }
    if (!ok)  // given up: the copies under way land before this CTA's shared memory is anyone else's
      for (int b = 0; b < S && b < i; ++b) {
        const long long start = clock64();
        while (!mbar_try_wait(smem_u32(full + b), b < slot ? phase : phase ^ 1) && clock64() - start < WAIT_CLOCKS) {
        }
      }
  } else if (warp == HP_WARP_MMA && n_tiles) {
    const uint32_t idesc_s = umma_idesc_bf16(HP_KEYS, false, false), idesc_o = umma_idesc_bf16(p.nv, false, true);
    const uint64_t dq0 = umma_smem_desc(sQ, 16, 1024), dk0 = umma_smem_desc(sKV, 16, 1024), dv0 = umma_smem_desc(sKV + p.ck * HP_K_CHUNK, HP_K_CHUNK, 1024);
    const uint32_t q_group = (uint32_t)p.q_bytes >> 4, stage = stage_bytes >> 4;
    const int nk = (a.dim + 15) / 16;
    int slot_s = 0, slot_v = 0;  // the ring's places of the scores' tile and of the sums'
    uint32_t phase_s = 0;
    auto scores = [&](int gr, int t) {
      const uint64_t dq = dq0 + gr * q_group, dk = dk0 + slot_s * stage;
      const uint32_t to = tmem + gr * HP_COLS + (t & 1) * HP_KEYS;
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        if (j >= nk) break;
        umma_bf16_warp(to, dq + (j >> 2) * (HP_Q_CHUNK >> 4) + 2 * (j & 3), dk + (j >> 2) * (HP_K_CHUNK >> 4) + 2 * (j & 3), idesc_s, j);
      }
      umma_commit_warp(smem_u32(s_full + 2 * gr + (t & 1)));
    };
    mbar_wait(smem_u32(full), 0, abort_flag, PW_FULL);
#pragma unroll
    for (int gr = 0; gr < GROUPS; ++gr) {
      mbar_wait(smem_u32(q_full + gr), 0, abort_flag, PW_Q);
      tc_fence_after();
      scores(gr, 0);
    }
    for (int t = 0; t < n_tiles; ++t) {
      if (t + 1 < n_tiles) {
        if (++slot_s == S) slot_s = 0, phase_s ^= 1;
        mbar_wait(smem_u32(full + slot_s), phase_s, abort_flag, PW_FULL);
      }
#pragma unroll
      for (int gr = 0; gr < GROUPS; ++gr) {
        if (t + 1 < n_tiles) {
          // (the buffer holds the probabilities of the tile before this one until their MMAs are done)
          if (t > 0) mbar_wait(smem_u32(pv_done + gr), (t - 1) & 1, abort_flag, PW_PV_MMA);
          tc_fence_after();
          scores(gr, t + 1);
        }
        mbar_wait(smem_u32(p_full + gr), t & 1, abort_flag, PW_P);
        tc_fence_after();
        const uint32_t tP = tmem + gr * HP_COLS + (t & 1) * HP_KEYS, tO = tmem + gr * HP_COLS + 2 * HP_KEYS;
        const uint64_t dv = dv0 + slot_v * stage;
#pragma unroll
        for (int kk = 0; kk < HP_KEYS / 16; ++kk) umma_bf16_ts_warp(tO, tP + 8 * kk, dv + kk * (2048 >> 4), idesc_o, t | kk);
        if (gr == GROUPS - 1) umma_commit_warp(smem_u32(empty + slot_v));
        umma_commit_warp(smem_u32(pv_done + gr));
      }
      if (++slot_v == S) slot_v = 0;
    }
  } else if (warp < 4 * GROUPS) {
    const int gr = warp >> 2, row = 32 * (warp & 3) + lane, head = g * a.rep + row % a.rep;
    const int64_t token = t0 + gr * p.tokens + row / a.rep;
    const bool live = row < p.tokens * a.rep && token < a.T;
    // (a row past the last runs along and is never looked at)
    const int place = live ? min(a.last[token], len - 1) : 0x3fffffff, first = live ? first_seen(a, a.last[token]) : 0;
    const uint32_t lanes = (uint32_t)(32 * (warp & 3)) << 16, tS = tmem + lanes + gr * HP_COLS, tO = tS + 2 * HP_KEYS;
    const float scale_log2 = a.scale * HP_LOG2E;
    const SoftCap cap = soft_cap(a);
    const float bias = SIGMOID && live ? a.key_bias[head] * HP_LOG2E : 0.f;
    float m = -INFINITY, l = 0.f;  // the reference maximum of the unscaled scores, and the sum under it
    for (int t = 0; t < n_tiles; ++t) {
      mbar_wait(smem_u32(s_full + 2 * gr + (t & 1)), (t >> 1) & 1, abort_flag, PW_S);
      tc_fence_after();
      if constexpr (SIGMOID) {  // 32 keys at a time over the columns read before, in a loop that stays in the instruction cache
        const int seen = place + 1 - (k0 + t * HP_KEYS), hidden = first - (k0 + t * HP_KEYS);
        const bool whole = __all_sync(0xffffffffu, seen >= HP_KEYS && hidden <= 0);
#pragma unroll 1
        for (int b = 0; b < HP_KEYS; b += 32) {
          float s[32], p[16];
          tmem_ld32_nowait(tS + (t & 1) * HP_KEYS + b, s);
          tmem_ld_wait();
          if (cap.in > 0.f) {
#pragma unroll
            for (int j = 0; j < 32; ++j) s[j] = capped(cap, s[j]);
          }
          if (!whole) {
#pragma unroll
            for (int j = 0; j < 32; ++j)
              if (b + j >= seen || b + j < hidden) s[j] = -INFINITY;
          }
#pragma unroll
          for (int j = 0; j < 32; j += 2) {
            float x, y;
            sigmoid_pair(fmaf(s[j], scale_log2, bias), fmaf(s[j + 1], scale_log2, bias), x, y);
            p[j / 2] = __uint_as_float(pack_bf16x2(s[j] == -INFINITY ? 0.f : x, s[j + 1] == -INFINITY ? 0.f : y));
          }
          tmem_st16(tS + (t & 1) * HP_KEYS + b / 2, p);
        }
        tmem_st_wait();
        if (t > 0) mbar_wait(smem_u32(pv_done + gr), (t - 1) & 1, abort_flag, PW_PV);  // (each tile's in turn: a phase two on looks like this one)
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(p_full + gr));
        continue;
      }
      float s[HP_KEYS];
      tmem_ld32_nowait(tS + (t & 1) * HP_KEYS, s);
      tmem_ld32_nowait(tS + (t & 1) * HP_KEYS + 32, s + 32);
      tmem_ld_wait();
      if (cap.in > 0.f) {
#pragma unroll
        for (int j = 0; j < HP_KEYS; ++j) s[j] = capped(cap, s[j]);
      }
      const int key0 = k0 + t * HP_KEYS, seen = place + 1 - key0, hidden = first - key0;  // of these keys, from `hidden` on and before `seen`
      if (!__all_sync(0xffffffffu, seen >= HP_KEYS && hidden <= 0)) {
#pragma unroll
        for (int j = 0; j < HP_KEYS; ++j)
          if (j >= seen || j < hidden) s[j] = -INFINITY;
      }
      float tops[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int j = 4; j < HP_KEYS; ++j) tops[j & 3] = fmaxf(tops[j & 3], s[j]);
      const float top = fmaxf(fmaxf(tops[0], tops[1]), fmaxf(tops[2], tops[3]));
      float corr = 1.f;
      const bool grown = (top - m) * scale_log2 > HP_SLACK || (m == -INFINITY && top > m);
      if (grown) corr = exp2_of((m - top) * scale_log2), m = top;
      const bool any = __any_sync(0xffffffffu, grown);
      const float at = m == -INFINITY ? 0.f : -m * scale_log2;
      float sums[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t pair[HP_KEYS / 2];
#pragma unroll
      for (int j = 0; j < HP_KEYS; j += 2) {
        const float x = exp2_of(fmaf(s[j], scale_log2, at)), y = exp2_of(fmaf(s[j + 1], scale_log2, at));
        sums[j & 2] += x, sums[(j & 2) + 1] += y;
        pair[j / 2] = pack_bf16x2(x, y);
      }
      l = l * corr + ((sums[0] + sums[1]) + (sums[2] + sums[3]));
      if (t > 0) {  // the sums stand still once the last tile's MMAs are done
        mbar_wait(smem_u32(pv_done + gr), (t - 1) & 1, abort_flag, PW_PV);
        tc_fence_after();
        if (any) {
          for (int c = 0; c < p.nv; c += 16) {
            float v[16];
            tmem_ld16_nowait(tO + c, v);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 16; ++e) v[e] *= corr;
            tmem_st16(tO + c, v);
          }
        }
      }
      tmem_st32(tS + (t & 1) * HP_KEYS, pair);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(p_full + gr));
    }
    // the result: 32 columns at a time through shared memory (the group's queries are done with), so that gates are read and
    // rows written across the columns
    float f = 0.f;
    if (live) {
      float total = l;
      f = 1.f;
      const float mine = m * scale_log2;
      if (a.sink) {
        const float sink = a.sink[head] * HP_LOG2E, top = fmaxf(mine, sink);
        f = exp2_of(mine - top), total = l * f + exp2_of(sink - top);
      }
      f = SIGMOID ? a.out_scale : total > 0.f ? f * a.out_scale / total : 0.f;
    }
    if (n_tiles) {
      mbar_wait(smem_u32(pv_done + gr), (n_tiles - 1) & 1, abort_flag, PW_PV);
      tc_fence_after();
    }
    const int64_t gate_at = token * a.ld_g + (int64_t)head * a.vdim, out_at = live ? token * a.ld_o + (int64_t)head * a.vdim : -1;
    float* stage = reinterpret_cast<float*>(smem + gr * p.q_bytes) + (warp & 3) * 32 * 33;
    for (int c = 0; c < a.vdim; c += 32) {
      float v[32];
      if (n_tiles) {
        tmem_ld16_nowait(tO + c, v);
        if (c + 16 < p.nv) tmem_ld16_nowait(tO + c + 16, v + 16);
        tmem_ld_wait();
      }
#pragma unroll
      for (int e = 0; e < 32; ++e) stage[lane * 33 + e] = n_tiles && c + e < p.nv ? v[e] * f : 0.f;
      __syncwarp();
      if (p.fours) {  // eight lanes a row, four columns each: all of a block's gates on their way at once
        const int c4 = 4 * (lane & 7);
        const bool mine = c + c4 < a.vdim;
        float4 gate[8];
        int64_t from[8], to[8];
#pragma unroll
        for (int r = 0; r < 8; ++r) {
          from[r] = __shfl_sync(0xffffffffu, gate_at, 4 * r + (lane >> 3)) + c + c4;
          to[r] = __shfl_sync(0xffffffffu, out_at, 4 * r + (lane >> 3));
          if (!mine) to[r] = -1;
          gate[r] = make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (a.gate && a.gate_dtype == FB_FP32) {
#pragma unroll
          for (int r = 0; r < 8; ++r)
            if (to[r] >= 0) gate[r] = four(static_cast<const float*>(a.gate) + from[r]);
        } else if (a.gate) {
#pragma unroll
          for (int r = 0; r < 8; ++r)
            if (to[r] >= 0) gate[r] = four(static_cast<const uint16_t*>(a.gate) + from[r]);
        }
#pragma unroll
        for (int r = 0; r < 8; ++r)
          if (to[r] >= 0) {
            const float* v = stage + (4 * r + (lane >> 3)) * 33 + c4;
            float4 y = make_float4(v[0], v[1], v[2], v[3]);
            if (a.gate) y = make_float4(gated(y.x, gate[r].x), gated(y.y, gate[r].y), gated(y.z, gate[r].z), gated(y.w, gate[r].w));
            put_four(static_cast<uint16_t*>(a.out) + to[r] + c + c4, y);
          }
        __syncwarp();
        continue;
      }
      const bool mine = c + lane < a.vdim;
#pragma unroll 1
      for (int r0 = 0; r0 < 32; r0 += 8) {
        float gate[8];
        int64_t to[8];
#pragma unroll
        for (int r = 0; r < 8; ++r) {  // (all on their way before the first is needed)
          const int64_t from = __shfl_sync(0xffffffffu, gate_at, r0 + r);
          to[r] = __shfl_sync(0xffffffffu, out_at, r0 + r);
          gate[r] = a.gate && mine && to[r] >= 0 ? gate_value(a, from + c + lane) : 0.f;
        }
#pragma unroll
        for (int r = 0; r < 8; ++r)
          if (mine && to[r] >= 0) {
            const float v = stage[(r0 + r) * 33 + lane];
            static_cast<uint16_t*>(a.out)[to[r] + c + lane] = (uint16_t)float_to_bf16_bits(a.gate ? gated(v, gate[r]) : v);
          }
      }
      __syncwarp();
    }
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (warp == HP_WARP_MMA) {
    tc_fence_after();
    tmem_dealloc(tmem, p.tmem_cols);
  }
}

// sizes of a launch with `groups` groups a CTA; false: shared memory does not take it
bool prompt_sizes(PromptParams& p, int groups) {
  const HeadsArgs& a = p.a;
  p.groups = groups, p.tokens = HP_ROWS / a.rep, p.ck = (a.dim + 63) / 64, p.cv = (a.vdim + 63) / 64, p.nv = (a.vdim + 15) / 16 * 16;
  p.q_bytes = p.ck * HP_Q_CHUNK > 17 * 1024 ? p.ck * HP_Q_CHUNK : 17 * 1024;  // (17 KB: what the result takes on its way out)
  p.tmem_cols = p.nv > 128 ? 512 : groups * HP_COLS;  // (sums of more than 128 columns: one group, all of tensor memory)
  if (p.nv > 128 && groups > 1) return false;
  const int64_t stage = (p.ck + p.cv) * HP_K_CHUNK, rest = 1024 + groups * p.q_bytes;
  p.smem = groups == 1 && p.nv <= 128 && rest + 2 * stage <= (int64_t)HP_SMEM_HALF ? HP_SMEM_HALF : HP_SMEM;
  const int64_t room = ((int64_t)p.smem - rest) / stage;
  p.stages = (int)(room < HP_MAX_STAGES ? room : HP_MAX_STAGES);
  return p.stages >= 2;
}

template <int GROUPS, bool SIGMOID>
int launch_prompt(const PromptParams& p, const CUtensorMap& tq, const CUtensorMap& tkv, cudaStream_t s) {
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(heads_prompt_kernel<GROUPS, SIGMOID>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)HP_SMEM);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3((unsigned)p.a.kv_heads, (unsigned)ceil_div(p.a.T, GROUPS * p.tokens)), cfg.blockDim = dim3((4 * GROUPS + 2) * 32);
  cfg.dynamicSmemBytes = p.smem, cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr, cfg.numAttrs = 1;
  cudaLaunchKernelEx(&cfg, heads_prompt_kernel<GROUPS, SIGMOID>, tq, tkv, p);
  return launch_status("fb_heads_attention");
}

}  // namespace

static const StatusWord g_status_reader(read_and_clear_status_word);

// a chunk of one sequence with tiles enough for half the SMs (fewer: heads_attention.cu splits the keys), heads that tensor
// memory takes, rows that TMA takes (the caller has checked that q and the cache are whole 16-byte pieces)
bool heads_prompt_supports(const HeadsArgs& a) {
  if (!a.chunk || a.rep > HP_ROWS || a.dim > 256 || a.vdim > 256 || a.ld_o % 2 || ceil_div(a.T, HP_ROWS / a.rep) > 65535 || a.cache_rows >= (1ll << 31)) return false;
  PromptParams p{};
  p.a = a;
  return ceil_div(a.T, HP_ROWS / a.rep) * a.kv_heads >= 74 && prompt_sizes(p, 1) && tma_encoder() != nullptr;
}

int heads_prompt(const HeadsArgs& a, cudaStream_t s) {
  PromptParams p{};
  p.a = a;
  // two groups a CTA share the tiles of wide heads; CTAs of narrow ones stand side by side on an SM instead
  const bool two = a.dim + a.vdim > 192 && ceil_div(a.T, 2 * (HP_ROWS / a.rep)) * a.kv_heads >= sm_count_of_device() && prompt_sizes(p, 2);
  if (!two) prompt_sizes(p, 1);
  p.fours = a.ld_o % 4 == 0 && (uintptr_t)a.out % 8 == 0 && (!a.gate || (a.ld_g % 4 == 0 && (uintptr_t)a.gate % (a.gate_dtype == FB_FP32 ? 16 : 8) == 0));
  CUtensorMap tq, tkv;
  const int64_t qd[4] = {a.dim, a.rep, a.kv_heads, a.T}, qs[3] = {a.dim, (int64_t)a.rep * a.dim, a.ld_q};
  const int qb[4] = {64, a.rep, 1, p.tokens};
  if (int rc = tma_map_bf16(&tq, a.q, 4, qd, qs, qb, "fb_heads_attention (queries)")) return rc;
  const int64_t kd[3] = {a.dim + a.vdim, a.cache_rows, a.kv_heads}, ks[2] = {a.dim + a.vdim, a.head_stride};
  const int kb[3] = {64, HP_KEYS, 1};
  if (int rc = tma_map_bf16(&tkv, a.cache, 3, kd, ks, kb, "fb_heads_attention (cache)")) return rc;
  if (a.key_bias) return two ? launch_prompt<2, true>(p, tq, tkv, s) : launch_prompt<1, true>(p, tq, tkv, s);
  return two ? launch_prompt<2, false>(p, tq, tkv, s) : launch_prompt<1, false>(p, tq, tkv, s);
}

}  // namespace fb
