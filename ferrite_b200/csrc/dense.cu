// fb_dense: activations by bf16 weights on the 5th-generation tensor cores, both operands by TMA.
//
// The weights are the MMA's A operand (a tile of 128 output columns = the 128 accumulator lanes in tensor memory), the
// tokens its N dimension (16 .. 256), so one kernel serves a decode step of a few tokens - bound by the stream of weights -
// and a prompt's hundreds, bound by the MMAs.  Both operands arrive K-major in 128-byte swizzled rows: no unpacking, no
// transposition, and the CTA's threads touch nothing but the accumulators.
//
//   warp 8      asks for the tiles: [128 x 64] of weights and [tokens x 64] of activations a step, a ring of 4 to 10 steps
//   warp 9      issues the MMAs (4 x K = 16 a step), one accumulator of two in tensor memory a tile
//   warps 0-7   the epilogue: a warp has a quarter of the lanes and half of the tokens; it empties one accumulator while the
//               MMAs fill the other
//
// CTAs are persistent: tiles are dealt out round robin, the ring and the accumulators run on across tile borders.  Where
// the tiles are too few to fill the GPU, K is split over the CTAs of a cluster (2, 4 or 8): each leaves its sums in shared
// memory, each then takes a share of the tokens and adds the others' sums to its own in rank order (the same every run).
//
// What follows a matmul in its model runs on the accumulators (fb_dense_epilogue): SiLU on the first columns, a squared
// ReLU, a clamped or a GELU-gated unit (gate and up rows alternate in runs of 16 inside a tile, so a pair is 16 lanes apart), a gate per head, and the
// Dynamic Tanh - residual add - Dynamic Tanh between two branches, which needs no sum over the row and therefore no
// kernel of its own.  Every wait is bounded (sm100.cuh).
//
// fb_dense_grouped is the same kernel over rows in tiles that each have a matrix of their own (a mixture's experts): which,
// and how many tiles there are, it reads on the device.
#include <math.h>

#include "sm100.cuh"
#include "tma_host.cuh"
#include "values.cuh"

namespace fb {

// whether W holds gate rows, then as many up rows, that meet in the epilogue
__host__ __device__ constexpr bool paired(int kind) { return kind == FB_DENSE_GLU || kind == FB_DENSE_GEGLU; }

namespace {

constexpr int D_EPI_WARPS = 8, D_WARP_LOAD = 8, D_WARP_MMA = 9, D_THREADS = 10 * 32;
constexpr int D_A_BYTES = 128 * 128;  // 128 weight rows of 64 values
constexpr int D_MAX_STAGES = 10;
constexpr size_t D_SMEM = 200 * 1024;

enum DenseWait { DW_EMPTY = 301, DW_FULL, DW_ACC_FULL, DW_ACC_EMPTY, DW_DRAIN };

struct DenseParams {
  int64_t M, N;  // N: output columns of W (gate and up together)
  int nt, stages, tmem_cols, steps, splits, steps_per_split;
  int tiles_m, tiles_n, tiles;  // tiles: all batch entries'
  void* out;
  int out_dtype;
  int64_t ldo, out_batch;
  int settled;
  // rows in tiles of `nt`, each with a matrix of its own (fb_dense_grouped): the tiles' matrices (and which tiles share one) and
  // how many there are, both read on the device; x_step: how far the rows move on a tile (nt, or 0: every tile the same rows)
  const int32_t *tile_expert, *live;
  int x_step;
  float shift;  // GLU: added to the up half
  fb_dense_epilogue e;
};

struct DenseTile {
  int m, n, b;
};
// tiles_m: the tiles of rows there are (grouped: those in use)
__device__ __forceinline__ DenseTile tile_of(const DenseParams& p, int id, int tiles_m) {  // tokens fastest: tiles that share weights run together
  if (p.tile_expert) {  // (a matrix after the other, so that its rows are read again from L2: the tiles id / tiles_n has them side by side)
    const int32_t* run = p.tile_expert + 3 * (id / p.tiles_n);
    const int at = id - run[1] * p.tiles_n;
    return {run[1] + at % run[2], at / run[2], run[0]};
  }
  const int rest = id / tiles_m;
  return {id % tiles_m, rest % p.tiles_n, rest / p.tiles_n};
}

// what the epilogue needs of a column, read once a tile
struct Column {
  float alpha, w, b, alpha2, w2, b2;
};
template <int EPI>
__device__ __forceinline__ Column column_of(const DenseParams& p, int64_t n, bool live) {
  Column c{};
  if constexpr (EPI == FB_DENSE_DYT_ADD) {
    if (live) {
      c.alpha = *p.e.alpha, c.w = p.e.w[n], c.b = p.e.b[n];
      if (p.e.h_out) c.alpha2 = *p.e.alpha2, c.w2 = p.e.w2[n], c.b2 = p.e.b2[n];
    }
  }
  if constexpr (EPI == FB_DENSE_GEGLU) {
    if (live) c.w = p.e.gate_bias ? p.e.gate_bias[n] : 0.f, c.b = p.e.up_bias ? p.e.up_bias[n] : 0.f;
  }
  return c;
}

// one value of the result: column n of token t (GLU: v the gate, up its partner); the caller has checked the bounds
template <int EPI>
__device__ __forceinline__ void emit(const DenseParams& p, const Column& c, int b, int64_t t, int64_t n, float v, float up, float res, float gate) {
  if constexpr (EPI == FB_DENSE_DYT_ADD) {
    const float x = res + fmaf(tanh_of(c.alpha * v), c.w, c.b);
    static_cast<float*>(p.out)[t * p.ldo + n] = x;
    if (p.e.h_out) static_cast<uint16_t*>(p.e.h_out)[t * p.e.ld_h + n] = (uint16_t)float_to_bf16_bits(fmaf(tanh_of(c.alpha2 * x), c.w2, c.b2));
    return;
  }
  if constexpr (EPI == FB_DENSE_SILU) {
    if (n < p.e.act_cols) v = __fdividef(v, 1.f + __expf(-v));
  }
  if constexpr (EPI == FB_DENSE_GLU || EPI == FB_DENSE_RELU2) {
    if (p.e.row_scale) {
      const float s = p.e.row_scale[t];
      v *= s, up *= s;
    }
  }
  if constexpr (EPI == FB_DENSE_RELU2) v = fmaxf(v, 0.f), v *= v;
  if constexpr (EPI == FB_DENSE_GLU) {
    const float g = fminf(v, p.e.limit), u = fminf(fmaxf(up, -p.e.limit), p.e.limit);
    v = g / (1.f + __expf(-p.e.slope * g)) * (u + p.shift);
  }
  if constexpr (EPI == FB_DENSE_GEGLU) {
    const float g = v + c.w;
    v = 0.5f * g * (1.f + tanh_of(0.7978845608028654f * fmaf(0.044715f * g * g, g, g))) * (up + c.b);
  }
  if constexpr (EPI == FB_DENSE_GATE) v *= gate;
  const int64_t at = b * p.out_batch + t * p.ldo + n;  // (grouped: out_batch 0, the rows follow the tiles)
  if (p.out_dtype == FB_FP32) static_cast<float*>(p.out)[at] = v;
  else static_cast<uint16_t*>(p.out)[at] = (uint16_t)float_to_bf16_bits(v);
}

template <int EPI>
__global__ void __launch_bounds__(D_THREADS, 1) dense_kernel(const __grid_constant__ CUtensorMap tw, const __grid_constant__ CUtensorMap tx, const DenseParams p) {
  extern __shared__ uint8_t dense_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(dense_smem) + 1023) & ~uintptr_t(1023));
  __shared__ uint64_t bars[2 * D_MAX_STAGES + 4];
  __shared__ uint32_t tmem_slot[2];  // the allocation's address, the abort flag
  uint64_t *full = bars, *empty = bars + D_MAX_STAGES, *acc_full = bars + 2 * D_MAX_STAGES, *acc_empty = acc_full + 2;
  const uint32_t abort_flag = smem_u32(tmem_slot + 1);
  const int tid = threadIdx.x, warp = uniform_warp(), lane = tid & 31;
  const int S = p.stages, nt = p.nt, stage_bytes = D_A_BYTES + nt * 128;
  const int s0 = blockIdx.y * p.steps_per_split, n_steps = min(p.steps - s0, p.steps_per_split);

  griddep_launch_dependents();
  if (tid == 0) {
    for (int s = 0; s < S; ++s) mbar_init(smem_u32(full + s), 1), mbar_init(smem_u32(empty + s), 1);
    for (int s = 0; s < 2; ++s) mbar_init(smem_u32(acc_full + s), 1), mbar_init(smem_u32(acc_empty + s), D_EPI_WARPS);
    tmem_slot[1] = 0;
    fence_barrier_init();
  }
  if (warp == D_WARP_MMA) tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot[0];
  int tiles = p.tiles, tiles_m = p.tiles_m;
  if (p.live) {
    griddep_wait();
    tiles_m = min(max(*p.live, 0), p.tiles_m), tiles = tiles_m * p.tiles_n;
  }
  const bool idle = p.splits > 1 && (int)blockIdx.x >= tiles;  // (a whole cluster without a tile)

  if (warp == D_WARP_LOAD && lane == 0) {
    prefetch_tensormap(&tw), prefetch_tensormap(&tx);
    auto weights = [&](const DenseTile& t, int k, int slot) {
      const uint32_t bar = smem_u32(full + slot), dst = smem_u32(smem + slot * stage_bytes);
      mbar_expect_tx(bar, (uint32_t)stage_bytes);
      if (paired(EPI)) tma_load_5d(dst, &tw, 64 * k, 0, 0, 4 * t.n, t.b, bar);
      else tma_load_3d(dst, &tw, 64 * k, 128 * t.n, t.b, bar);
    };
    int early = 0;
    if (p.settled && !p.live && (int)blockIdx.x < p.tiles) {
      const DenseTile t = tile_of(p, blockIdx.x, tiles_m);
      for (early = 0; early < min(S, n_steps); ++early) weights(t, s0 + early, early);
    }
    griddep_wait();  // the activations come from the kernel before
    int i = 0, slot = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (int id = blockIdx.x; id < tiles && ok; id += gridDim.x) {
      const DenseTile t = tile_of(p, id, tiles_m);
      for (int k = 0; k < n_steps && ok; ++k, ++i) {
        if (i >= early) {
          ok = mbar_wait(smem_u32(empty + slot), phase ^ 1, abort_flag, DW_EMPTY);
          if (!ok) break;
          weights(t, s0 + k, slot);
        }
        tma_load_3d(smem_u32(smem + slot * stage_bytes + D_A_BYTES), &tx, 64 * (s0 + k), p.x_step * t.m, p.live ? 0 : t.b, smem_u32(full + slot));
        if (++slot == S) slot = 0, phase ^= 1;
      }
    }
    if (!ok)  // given up: the copies under way land before this CTA's shared memory is anyone else's
      for (int s = 0; s < S; ++s) {
        const long long start = clock64();
        const uint32_t parity = s < slot ? phase : phase ^ 1;
        while (i > s && !mbar_try_wait(smem_u32(full + s), parity) && clock64() - start < WAIT_CLOCKS) {
        }
      }
  } else if (warp == D_WARP_MMA) {
    const uint32_t idesc = umma_idesc_bf16(nt, false, false);
    const uint64_t d0 = umma_smem_desc(smem_u32(smem), 16, 1024);
    int slot = 0, n = 0;
    uint32_t phase = 0;
    for (int id = blockIdx.x; id < tiles; id += gridDim.x, ++n) {
      const uint32_t acc = tmem + (n & 1) * nt;
      mbar_wait(smem_u32(acc_empty + (n & 1)), ((n >> 1) & 1) ^ 1, abort_flag, DW_ACC_EMPTY);
      tc_fence_after();
      for (int k = 0; k < n_steps; ++k) {
        mbar_wait(smem_u32(full + slot), phase, abort_flag, DW_FULL);
        tc_fence_after();
        const uint64_t da = d0 + (uint32_t)(slot * stage_bytes >> 4), dx = da + (D_A_BYTES >> 4);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) umma_bf16_warp(acc, da + 2 * kk, dx + 2 * kk, idesc, k | kk);
        umma_commit_warp(smem_u32(empty + slot));
        if (++slot == S) slot = 0, phase ^= 1;
      }
      umma_commit_warp(smem_u32(acc_full + (n & 1)));
    }
  } else if (warp < D_EPI_WARPS) {
    griddep_wait();
    const int q = warp & 3, half = nt / 2, col0 = (warp >> 2) * half, row = 32 * q + lane;
    int n = 0;
    for (int id = blockIdx.x; id < tiles; id += gridDim.x, ++n) {
      const DenseTile t = tile_of(p, id, tiles_m);
      mbar_wait(smem_u32(acc_full + (n & 1)), (n >> 1) & 1, abort_flag, DW_ACC_FULL);
      tc_fence_after();
      const uint32_t acc = tmem + ((uint32_t)(32 * q) << 16) + (n & 1) * nt + col0;
      const int64_t t0 = (int64_t)nt * t.m + col0;
      if (p.splits > 1) {  // this CTA's part of the sums, token by token, for the cluster to read
        float* ex = reinterpret_cast<float*>(smem);
        for (int c = 0; c < half; c += 8) {
          float v[8];
          tmem_ld8(acc + c, v);
#pragma unroll
          for (int e = 0; e < 8; ++e) ex[(col0 + c + e) * 128 + row] = v[e];
        }
      } else {
        const int64_t col = paired(EPI) ? 64 * (int64_t)t.n + 16 * q + (lane & 15) : 128 * (int64_t)t.n + row;
        const bool live = col < (paired(EPI) ? p.N / 2 : p.N);
        const Column mine = column_of<EPI>(p, col, live);
        for (int c = 0; c < half && t0 + c < p.M; c += 8) {
          float v[8], extra[8];
          tmem_ld8_nowait(acc + c, v);
          if constexpr (EPI == FB_DENSE_DYT_ADD || EPI == FB_DENSE_GATE) {
#pragma unroll
            for (int e = 0; e < 8; ++e) {
              const int64_t tt = t0 + c + e;
              extra[e] = 0.f;
              if (tt < p.M && live) extra[e] = EPI == FB_DENSE_GATE ? p.e.gate[tt * p.e.ld_gate + t.b] : p.e.residual[tt * p.e.ld_residual + col];
            }
          }
          tmem_ld_wait();
          if constexpr (paired(EPI)) {
            // lanes 0-15 hold gates, 16-31 their ups: the low half takes the first four tokens, the high half the others
            const bool high = lane >= 16;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float got = __shfl_xor_sync(0xffffffffu, high ? v[e] : v[e + 4], 16);
              const int64_t tt = t0 + c + e + (high ? 4 : 0);
              if (tt < p.M && live) emit<EPI>(p, mine, t.b, tt, col, high ? got : v[e], high ? v[e + 4] : got, 0.f, 0.f);
            }
          } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) {
              const int64_t tt = t0 + c + e;
              if (tt < p.M && live) {
                if constexpr (EPI == FB_DENSE_GATE) emit<EPI>(p, mine, t.b, tt, col, v[e], 0.f, 0.f, 1.f / (1.f + __expf(-extra[e])));
                else emit<EPI>(p, mine, t.b, tt, col, v[e], 0.f, EPI == FB_DENSE_DYT_ADD ? extra[e] : 0.f, 0.f);
              }
            }
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(acc_empty + (n & 1)));
    }
  }
  __syncwarp();

  if (p.splits > 1) {
    cluster_barrier();  // every CTA's sums are in its shared memory
    if (warp < D_EPI_WARPS && !idle) {
      const DenseTile t = tile_of(p, blockIdx.x, tiles_m);
      const int share = (nt + p.splits - 1) / p.splits, first = blockIdx.y * share, last = min(nt, first + share);
      const int row = tid & 127;
      const int64_t col = paired(EPI) ? 64 * (int64_t)t.n + (row >> 5) * 16 + (row & 15) : 128 * (int64_t)t.n + row;
      const bool live = col < (paired(EPI) ? p.N / 2 : p.N) && (!paired(EPI) || !(row & 16));
      const Column mine = column_of<EPI>(p, col, live);
      for (int c = first + (tid >> 7); c < last; c += 2) {
        const int64_t tt = (int64_t)nt * t.m + c;
        if (tt >= p.M || !live) continue;
        const uint32_t at = smem_u32(smem) + (uint32_t)(c * 128 + row) * 4;
        float v = 0.f, up = 0.f, res = 0.f, gate = 0.f;
        if constexpr (EPI == FB_DENSE_DYT_ADD) res = p.e.residual[tt * p.e.ld_residual + col];
        if constexpr (EPI == FB_DENSE_GATE) gate = 1.f / (1.f + __expf(-p.e.gate[tt * p.e.ld_gate + t.b]));
        float part[8], upper[8];  // (all on their way before the first is needed)
#pragma unroll
        for (int s = 0; s < 8; ++s) {
          part[s] = upper[s] = 0.f;
          if (s < p.splits) {
            part[s] = load_cluster_f32(at, s);
            if constexpr (paired(EPI)) upper[s] = load_cluster_f32(at + 64, s);
          }
        }
#pragma unroll
        for (int s = 0; s < 8; ++s) v += part[s], up += upper[s];
        emit<EPI>(p, mine, t.b, tt, col, v, up, res, gate);
      }
    }
    cluster_barrier();  // the others have read what they need of this CTA's shared memory
  }
  __syncthreads();
  if (warp == D_WARP_MMA) {
    tc_fence_after();
    tmem_dealloc(tmem, p.tmem_cols);
  }
}

template <int EPI>
int launch_dense(const CUtensorMap& tw, const CUtensorMap& tx, const DenseParams& p, int grid, size_t smem, cudaStream_t s) {
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(dense_kernel<EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3((unsigned)grid, (unsigned)p.splits), cfg.blockDim = dim3(D_THREADS), cfg.dynamicSmemBytes = smem, cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = 1, attr[1].val.clusterDim.y = (unsigned)p.splits, attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr, cfg.numAttrs = p.splits > 1 ? 2 : 1;
  cudaLaunchKernelEx(&cfg, dense_kernel<EPI>, tw, tx, p);
  return launch_status("fb_dense");
}

}  // namespace

static const StatusWord g_status_reader(read_and_clear_status_word);

}  // namespace fb

extern "C" int fb_dense_supports(const void* x, int64_t ldx, int64_t x_batch, const void* W, int64_t ldw, int64_t w_batch, int64_t K, int64_t N, int kind) {
  return K >= 8 && K % 8 == 0 && N >= 1 && ldx % 8 == 0 && ldw % 8 == 0 && x_batch % 8 == 0 && w_batch % 8 == 0 && ldx >= K && ldw >= K && (uintptr_t)x % 16 == 0 &&
         (uintptr_t)W % 16 == 0 && ((!fb::paired(kind) && kind != FB_DENSE_SWIGLU) || N % 32 == 0) && fb::tma_encoder() != nullptr;
}

// what fb_dense and fb_dense_grouped share: the tiles' depth and the CTAs', and the launch.  p: sizes, results and the way rows
// become tiles are filled in; x_rows, x_entries: the rows and batch entries that x has
static int run_dense(fb::DenseParams& p, const void* x, int64_t x_rows, int64_t x_entries, int64_t K, int64_t ldx, int64_t x_batch, const void* W, int64_t ldw, int64_t w_batch,
                     int64_t matrices, cudaStream_t s) {
  using namespace fb;
  const int kind = p.e.kind;
  p.steps = (int)ceil_div(K, 64);
  p.tmem_cols = 32;
  while (p.tmem_cols < 2 * p.nt) p.tmem_cols *= 2;
  const int stage_bytes = D_A_BYTES + p.nt * 128;
  p.stages = (int)(D_SMEM / stage_bytes);
  p.stages = p.stages > D_MAX_STAGES ? D_MAX_STAGES : p.stages;
  // K over the CTAs of a cluster where the tiles alone leave SMs idle: the split with the least modelled time
  const int sms = sm_count_of_device();
  p.splits = 1;
  double best = 1e30;
  for (int s = 1; s <= 8; s *= 2) {
    if (s > 1 && (p.tiles * s > (s == 8 ? 128 : sms) || p.steps < 2 * s)) break;  // (one round: clusters of eight leave some SMs unused)
    const int per = (int)ceil_div(p.steps, s);
    if ((int)ceil_div(p.steps, per) != s) continue;
    const double step = 0.12 + 0.001 * p.nt + 0.25 * (double)(p.tiles * s < sms ? p.tiles * s : sms) / sms;  // us: latency-bound at first, then the stream's share
    const double cost = (double)ceil_div((int64_t)p.tiles * s, sms) * (per * step + 0.5) + (s > 1 ? 1.0 : 0.0);
    if (cost < best) best = cost, p.splits = s;
  }
  p.steps_per_split = (int)ceil_div(p.steps, p.splits);
  const int grid = p.splits > 1 ? p.tiles : p.tiles < sms ? p.tiles : sms;
  CUtensorMap tw, tx;
  if (paired(kind)) {
    const int64_t dims[5] = {K, 16, 2, p.N / 32, matrices}, strides[4] = {ldw, p.N / 2 * ldw, 16 * ldw, matrices > 1 ? w_batch : ldw};
    const int box[5] = {64, 16, 2, 4, 1};
    if (int rc = tma_map_bf16(&tw, W, 5, dims, strides, box, "fb_dense (weights)")) return rc;
  } else {
    const int64_t dims[3] = {K, p.N, matrices}, strides[2] = {ldw, matrices > 1 ? w_batch : ldw};
    const int box[3] = {64, 128, 1};
    if (int rc = tma_map_bf16(&tw, W, 3, dims, strides, box, "fb_dense (weights)")) return rc;
  }
  const int64_t dims[3] = {K, x_rows, x_entries}, strides[2] = {ldx, x_entries > 1 && x_batch ? x_batch : ldx};
  const int box[3] = {64, p.nt, 1};
  if (int rc = tma_map_bf16(&tx, x, 3, dims, strides, box, "fb_dense (activations)")) return rc;
  const size_t smem = 1024 + (size_t)p.stages * stage_bytes;
  switch (kind) {
    case FB_DENSE_SILU: return launch_dense<FB_DENSE_SILU>(tw, tx, p, grid, smem, s);
    case FB_DENSE_GLU: return launch_dense<FB_DENSE_GLU>(tw, tx, p, grid, smem, s);
    case FB_DENSE_GEGLU: return launch_dense<FB_DENSE_GEGLU>(tw, tx, p, grid, smem, s);
    case FB_DENSE_RELU2: return launch_dense<FB_DENSE_RELU2>(tw, tx, p, grid, smem, s);
    case FB_DENSE_GATE: return launch_dense<FB_DENSE_GATE>(tw, tx, p, grid, smem, s);
    case FB_DENSE_DYT_ADD: return launch_dense<FB_DENSE_DYT_ADD>(tw, tx, p, grid, smem, s);
    default: return launch_dense<FB_DENSE_NONE>(tw, tx, p, grid, smem, s);
  }
}

// FB_DENSE_SWIGLU is the clamped unit without its limit, slope and shift
static float settle_unit(fb_dense_epilogue& e) {
  if (e.kind != FB_DENSE_SWIGLU) return 1.f;
  e.kind = FB_DENSE_GLU, e.limit = INFINITY, e.slope = 1.f;
  return 0.f;
}

extern "C" int fb_dense(const void* x, int64_t M, int64_t K, int64_t ldx, int64_t x_batch, const void* W, int64_t N, int64_t ldw, int64_t w_batch, int64_t batch,
                        void* out, int out_dtype, int64_t ldo, int64_t out_batch, const fb_dense_epilogue* epilogue_host, int settled, void* stream) {
  using namespace fb;
  FB_REQUIRE(x && W && out && M >= 1 && batch >= 1 && M < (1 << 30) && N < (1 << 30), "fb_dense: null pointer or empty");
  fb_dense_epilogue e = epilogue_host ? *epilogue_host : fb_dense_epilogue{};
  FB_REQUIRE(e.kind >= FB_DENSE_NONE && e.kind <= FB_DENSE_RELU2, "fb_dense: unknown epilogue %d", e.kind);
  const float shift = settle_unit(e);
  FB_REQUIRE(K >= 8 && K % 8 == 0 && ldx % 8 == 0 && ldw % 8 == 0 && x_batch % 8 == 0 && w_batch % 8 == 0 && ldx >= K && ldw >= K && (uintptr_t)x % 16 == 0 &&
                 (uintptr_t)W % 16 == 0 && N >= 1,
             "fb_dense: rows of x and W 16-byte aligned, K a multiple of 8 (K %lld, row strides %lld and %lld)", (long long)K, (long long)ldx, (long long)ldw);
  FB_REQUIRE(out_dtype == FB_BF16 || out_dtype == FB_FP32, "fb_dense: out is bf16 or fp32");
  FB_REQUIRE(!paired(e.kind) || (N % 32 == 0 && batch == 1), "fb_dense: a gated unit takes one matrix of whole runs of 16 gate rows and as many up rows");
  FB_REQUIRE(e.kind != FB_DENSE_GATE || e.gate, "fb_dense: no gate given");
  FB_REQUIRE(e.kind != FB_DENSE_DYT_ADD || (e.residual && e.alpha && e.w && e.b && out_dtype == FB_FP32 && batch == 1 && (!e.h_out || (e.alpha2 && e.w2 && e.b2))),
             "fb_dense: a Dynamic Tanh and add takes its vectors, a residual and an fp32 result");
  FB_REQUIRE(tma_encoder() != nullptr, "fb_dense: no CUDA driver");
  const int64_t out_cols = fb::paired(e.kind) ? N / 2 : N;
  FB_REQUIRE(ldo >= out_cols, "fb_dense: rows of out too close");
  DenseParams p{};
  p.M = M, p.N = N, p.e = e, p.out = out, p.out_dtype = out_dtype, p.ldo = ldo, p.out_batch = out_batch, p.settled = settled, p.shift = shift;
  p.tiles_m = (int)ceil_div(M, 256);
  p.nt = (int)ceil_div(ceil_div(M, p.tiles_m), 16) * 16;
  p.tiles_m = (int)ceil_div(M, p.nt);
  p.tiles_n = (int)ceil_div(out_cols, fb::paired(e.kind) ? 64 : 128);
  FB_REQUIRE((int64_t)p.tiles_m * p.tiles_n * batch < (1 << 30), "fb_dense: too many tiles");
  p.tiles = (int)(p.tiles_m * p.tiles_n * batch);
  p.x_step = p.nt;
  FB_REQUIRE(batch == 1 || x_batch > 0, "fb_dense: a batch takes rows of its own an entry");
  return run_dense(p, x, M, batch, K, ldx, x_batch, W, ldw, w_batch, batch, (cudaStream_t)stream);
}

extern "C" int fb_dense_grouped(const void* x, int64_t x_rows, int64_t K, int64_t ldx, int shared_rows, const void* W, int64_t N, int64_t ldw, int64_t w_batch, int n,
                                const int32_t* tile_expert, const int32_t* live, int64_t tiles, int tile, void* out, int out_dtype, int64_t ldo,
                                const fb_dense_epilogue* epilogue_host, void* stream) {
  using namespace fb;
  FB_REQUIRE(x && W && out && tile_expert && live && tiles >= 1 && n >= 1 && x_rows >= 1 && tiles * tile < (1 << 30) && N < (1 << 30), "fb_dense_grouped: null pointer or empty");
  fb_dense_epilogue e = epilogue_host ? *epilogue_host : fb_dense_epilogue{};
  FB_REQUIRE(e.kind == FB_DENSE_NONE || e.kind == FB_DENSE_GLU || e.kind == FB_DENSE_SWIGLU || e.kind == FB_DENSE_RELU2, "fb_dense_grouped: plain, a gated unit or a squared ReLU");
  FB_REQUIRE(!e.row_scale || e.kind != FB_DENSE_NONE, "fb_dense_grouped: weights on the input of a unit take one");
  FB_REQUIRE(tile >= 16 && tile <= 256 && tile % 16 == 0 && (shared_rows ? x_rows <= tile : x_rows >= tiles * tile), "fb_dense_grouped: tiles of 16 to 256 rows, all of them there");
  FB_REQUIRE(fb_dense_supports(x, ldx, 0, W, ldw, n > 1 ? w_batch : 0, K, N, e.kind), "fb_dense_grouped: rows of x and W 16-byte aligned, K a multiple of 8, a gated unit's halves whole runs of 16");
  FB_REQUIRE(out_dtype == FB_BF16 || out_dtype == FB_FP32, "fb_dense_grouped: out is bf16 or fp32");
  DenseParams p{};
  p.shift = settle_unit(e);
  const int64_t out_cols = fb::paired(e.kind) ? N / 2 : N;
  FB_REQUIRE(ldo >= out_cols, "fb_dense_grouped: rows of out too close");
  p.M = tiles * tile, p.N = N, p.e = e, p.out = out, p.out_dtype = out_dtype, p.ldo = ldo;
  p.nt = tile, p.tiles_m = (int)tiles, p.x_step = shared_rows ? 0 : tile, p.tile_expert = tile_expert, p.live = live;
  p.tiles_n = (int)ceil_div(out_cols, fb::paired(e.kind) ? 64 : 128);
  FB_REQUIRE(tiles * p.tiles_n < (1 << 30), "fb_dense_grouped: too many tiles");
  p.tiles = (int)tiles * p.tiles_n;
  return run_dense(p, x, x_rows, 1, K, ldx, 0, W, ldw, w_batch, n, (cudaStream_t)stream);
}
