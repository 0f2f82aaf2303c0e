// fb_latent_attention on the 5th-generation tensor cores (bf16 rows).
//
// All heads of a token read the same cache row, and one row is key and value at once, so the unit of work is a tile of up
// to 64 query ROWS - (token, head) pairs that see keys of one sequence: a decode step's heads of a token, or consecutive
// pairs of a prompt's chunk - by tiles of KT cache rows (64, 48 or 32: what leaves room for three tiles), each brought in by
// TMA once and used twice from shared memory:
//
//   scores    S [rows, KT keys]    = Q [rows, W] . K^T       Q is the MMA's A operand (its 128 lanes read past the last row: lanes
//                                                            of no row, never looked at), the keys its N
//   sums      O^T [128 columns of the latent, rows] += V^T P^T   the same tile of cache rows as A operand, now with the
//                                                            latent's columns as lanes; P from shared memory as B
//
// so a softmax thread owns a row's scores (tcgen05.ld; two threads agree on a row's maximum, nothing else is exchanged), and the sums of a
// 512-column latent by 64 rows take half of tensor memory.  The sums stand under a reference maximum that moves only when a
// row's scores outgrow it by a factor of 256; then (rarely after the first tiles) the accumulators are rescaled.
//
//   warps 0-7   softmax (two warps share 32 rows, half a tile's keys each); rescaling; the result
//   warp 8      TMA          warp 9   MMAs (the whole warp issues them, written out: a loop around each, or one lane alone, would cost more than the MMA)
//
// With three tiles or more in the ring the next tile's scores are computed while this tile's softmax runs.  Few row tiles are split along the keys over more CTAs: up to eight as a cluster, whose parts stay in
// shared memory and are merged there, each CTA a share of the rows; beyond that through global memory and
// latent_combine_kernel.  The sink is one more part with a maximum and no value.  Every wait is bounded (sm100.cuh).
#include "latent.cuh"
#include "sm100.cuh"
#include "tma_host.cuh"

namespace fb {

namespace {

constexpr int L_ROWS = 64, L_WARP_LOAD = 8, L_WARP_MMA = 9, L_SOFTMAX = 256, L_THREADS = 10 * 32, L_MAX_BUFS = 4;
constexpr size_t L_SMEM = 225 * 1024;
constexpr int L_MAX_CHUNKS = 9, L_MAX_BLOCKS = 4;  // rows of up to 576 columns, latents of up to 512
constexpr float L_SLACK = 8.f;  // log2 of how far scores may outgrow the reference maximum

enum LatentWait { LW_Q = 401, LW_K_EMPTY, LW_K_FULL, LW_S, LW_P, LW_PV, LW_DRAIN };

struct LatentParams {
  LatentArgs a;
  int nr, keys, chunks, blocks, bufs, tmem_cols, splits, clustered, tiles_per_token;  // tiles_per_token: 0 for a chunk (tiles run through its rows)
  float scale_log2;
  float *part_o, *part_ml;  // [tile, split, 64, rank] and [tile, split, 64, 2]
};

// a barrier of the softmax warps; true if any of their threads brings a true
__device__ __forceinline__ bool softmax_any(bool mine) {
  uint32_t any;
  asm volatile("{\n.reg .pred p, q;\nsetp.ne.u32 q, %1, 0;\nbarrier.cta.red.or.aligned.pred p, 1, 256, q;\nselp.u32 %0, 1, 0, p;\n}" : "=r"(any) : "r"((uint32_t)mine) : "memory");
  return any != 0;
}
__device__ __forceinline__ void softmax_sync() { asm volatile("barrier.cta.sync.aligned 1, 256;" ::: "memory"); }

__device__ __forceinline__ float exp2_fast(float x) {  // (0 from -infinity)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// rows as TMA sees them: their whole 64-column pieces as a third axis (all of them come in one copy), and the ragged last piece
struct LatentMaps {
  CUtensorMap q, k, q_tail, k_tail;
};

// where a row tile stands: its first (token, head) pair, how many, and the keys it reads
struct RowTile {
  int64_t first_row, seq_first;
  int rows, first_key, keys;  // keys first_key .. keys - 1
};
__device__ __forceinline__ int first_seen(const LatentArgs& a, int place) { return a.window > 0 ? max(0, place - a.window + 1) : 0; }
__device__ __forceinline__ RowTile row_tile(const LatentParams& p, int tile) {
  const LatentArgs& a = p.a;
  RowTile r;
  int t0, t1;  // (pairs, and so tokens, are fewer than 2^31)
  if (p.tiles_per_token) {
    t0 = t1 = tile / p.tiles_per_token;
    const int g = tile - t0 * p.tiles_per_token;
    r.first_row = (int64_t)t0 * a.heads + g * L_ROWS, r.rows = min(L_ROWS, a.heads - g * L_ROWS);
  } else {
    r.first_row = (int64_t)tile * L_ROWS, r.rows = (int)min((int64_t)L_ROWS, a.T * a.heads - r.first_row);
    t0 = (int)r.first_row / a.heads, t1 = ((int)r.first_row + r.rows - 1) / a.heads;
  }
  r.seq_first = (a.base ? a.base[t0] : 0) + a.row0;
  int last = -1, lo = 0x7fffffff;
  for (int t = t0; t <= t1; ++t) last = max(last, a.last[t]), lo = min(lo, first_seen(a, a.last[t]));
  const int64_t room = r.seq_first < 0 ? 0 : a.cache_rows - r.seq_first;
  r.keys = (int)max((int64_t)0, min((int64_t)last + 1, room)), r.first_key = max(0, min(lo, r.keys));
  return r;
}

template <int KT>  // cache rows a tile
__global__ void __launch_bounds__(L_THREADS, 1) latent_tcgen05_kernel(const __grid_constant__ LatentMaps maps, const LatentParams p) {
  constexpr int L_KEYS = KT, L_CHUNK = KT * 128, MINE = KT / 2;  // a tile, 64 columns of it, a softmax thread's keys
  extern __shared__ uint8_t latent_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(latent_smem) + 1023) & ~uintptr_t(1023));
  __shared__ uint64_t bars[2 * L_MAX_BUFS + 5];
  __shared__ uint32_t tmem_slot[2];  // the allocation's address, the abort flag
  __shared__ float row_scale[L_ROWS], row_top[2][2][L_ROWS];  // per row: a factor; each half's maximum, two tiles' of them
  uint64_t *k_full = bars, *k_empty = bars + L_MAX_BUFS, *q_full = bars + 2 * L_MAX_BUFS, *s_full = q_full + 1, *p_full = q_full + 3, *pv_done = q_full + 4;
  const uint32_t abort_flag = smem_u32(tmem_slot + 1);
  const LatentArgs& a = p.a;
  const int tid = threadIdx.x, warp = uniform_warp(), lane = tid & 31;
  const int nr = p.nr, C = p.chunks, NB = p.bufs;
  const int tile = p.tiles_per_token ? blockIdx.x : gridDim.x - 1 - blockIdx.x, split = blockIdx.y;  // (a chunk's longest rows first)
  const uint32_t sQ = smem_u32(smem), sK = sQ + C * nr * 128, tile_bytes = C * L_CHUNK, sP = sK + NB * tile_bytes;

  griddep_launch_dependents();
  if (tid == 0) {
    for (int i = 0; i < NB; ++i) mbar_init(smem_u32(k_full + i), 1), mbar_init(smem_u32(k_empty + i), 1);
    mbar_init(smem_u32(q_full), 1), mbar_init(smem_u32(s_full), 1), mbar_init(smem_u32(s_full + 1), 1);
    mbar_init(smem_u32(p_full), L_SOFTMAX / 32), mbar_init(smem_u32(pv_done), 1);
    tmem_slot[1] = 0;
    fence_barrier_init();
  }
  if (warp == L_WARP_MMA) tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot[0], tS = tmem, tO = tmem + 128;
  griddep_wait();

  const RowTile r = row_tile(p, tile);
  // this CTA's run of whole tiles of keys
  const int all = (r.keys - r.first_key + L_KEYS - 1) / L_KEYS, per = (all + p.splits - 1) / p.splits;
  const int first_tile = split * per, n_tiles = max(0, min(all, first_tile + per) - first_tile);

  if (warp == L_WARP_LOAD && lane == 0) {
    const int whole = (a.rank + a.rot) / 64;  // pieces of 64 columns without the ragged last
    if (n_tiles) {
      mbar_expect_tx(smem_u32(q_full), (uint32_t)(C * nr * 128));
      if (whole) tma_load_3d(sQ, &maps.q, 0, (int)r.first_row, 0, smem_u32(q_full));
      if (whole < C) tma_load_2d(sQ + whole * nr * 128, &maps.q_tail, 64 * whole, (int)r.first_row, smem_u32(q_full));
    }
    int buf = 0, i = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (; i < n_tiles; ++i) {
      ok = mbar_wait(smem_u32(k_empty + buf), phase ^ 1, abort_flag, LW_K_EMPTY);
      if (!ok) break;
      mbar_expect_tx(smem_u32(k_full + buf), tile_bytes);
      const int at = (int)(r.seq_first + r.first_key + (int64_t)(first_tile + i) * L_KEYS);
      if (whole) tma_load_3d(sK + buf * tile_bytes, &maps.k, 0, at, 0, smem_u32(k_full + buf));
      if (whole < C) tma_load_2d(sK + buf * tile_bytes + whole * L_CHUNK, &maps.k_tail, 64 * whole, at, smem_u32(k_full + buf));
      if (++buf == NB) buf = 0, phase ^= 1;
    }
    if (!ok)  // given up: the copies under way land before this CTA's shared memory is anyone else's
      for (int b = 0; b < NB && b < i; ++b) {
        const long long start = clock64();
        while (!mbar_try_wait(smem_u32(k_full + b), b < buf ? phase : phase ^ 1) && clock64() - start < WAIT_CLOCKS) {
        }
      }
  } else if (warp == L_WARP_MMA && n_tiles) {
    const uint32_t idesc_s = umma_idesc_bf16(L_KEYS, false, false), idesc_o = umma_idesc_bf16(nr, true, false);
    const uint64_t dq0 = umma_smem_desc(sQ, 16, 1024), dk0 = umma_smem_desc(sK, 16, 1024), dv0 = umma_smem_desc(sK, L_CHUNK, 1024), dp = umma_smem_desc(sP, 16, 1024);
    const uint32_t q_chunk = (uint32_t)(nr * 128) >> 4, k_chunk = L_CHUNK >> 4, k_tile = tile_bytes >> 4;
    int sbuf = 0;  // the ring's place of the next scores
    uint32_t sphase = 0;
    auto scores = [&](int t) {
      mbar_wait(smem_u32(k_full + sbuf), sphase, abort_flag, LW_K_FULL);
      tc_fence_after();
      const uint64_t dk = dk0 + sbuf * k_tile;
      const uint32_t to = tS + (t & 1) * L_KEYS;
#pragma unroll
      for (int c = 0; c < L_MAX_CHUNKS; ++c) {
        if (c >= C) break;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) umma_bf16_warp(to, dq0 + c * q_chunk + 2 * kk, dk + c * k_chunk + 2 * kk, idesc_s, c | kk);
      }
      umma_commit_warp(smem_u32(s_full + (t & 1)));
      if (++sbuf == NB) sbuf = 0, sphase ^= 1;
    };
    mbar_wait(smem_u32(q_full), 0, abort_flag, LW_Q);
    scores(0);
    int vbuf = 0;
    for (int t = 0; t < n_tiles; ++t) {
      if (t + 1 < n_tiles) scores(t + 1);
      mbar_wait(smem_u32(p_full), t & 1, abort_flag, LW_P);
      tc_fence_after();
      const uint64_t dv = dv0 + vbuf * k_tile;
#pragma unroll
      for (int b = 0; b < L_MAX_BLOCKS; ++b) {
        if (b >= p.blocks) break;
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk)  // 16 keys each
          umma_bf16_warp(tO + b * nr, dv + 2 * b * k_chunk + kk * (2048 >> 4), dp + 2 * kk, idesc_o, t | kk);
      }
      umma_commit_warp(smem_u32(k_empty + vbuf));
      umma_commit_warp(smem_u32(pv_done));
      if (++vbuf == NB) vbuf = 0;
    }
  } else if (warp < L_SOFTMAX / 32) {
    const int half = warp >> 2, row = 32 * (warp & 3) + lane;  // lane `row` of the scores, half of a tile's keys (a lane past the last row runs along)
    const bool live = row < r.rows;
    const int place = live ? a.last[(r.first_row + row) / a.heads] : 0x3fffffff, first = live ? first_seen(a, place) : 0;
    const uint32_t lanes = (uint32_t)(32 * (warp & 3)) << 16;
    float m = -INFINITY, l = 0.f;  // the reference maximum (in units of log2) and this half's sum under it
    for (int t = 0; t < n_tiles; ++t) {
      mbar_wait(smem_u32(s_full + (t & 1)), (t >> 1) & 1, abort_flag, LW_S);
      tc_fence_after();
      float s[MINE];
      float top = -INFINITY;
      if (32 * (warp & 3) < nr) {
#pragma unroll
        for (int c = 0; c < MINE; c += 8) tmem_ld8_nowait(tS + lanes + (t & 1) * KT + MINE * half + c, s + c);
        tmem_ld_wait();
        const int key0 = r.first_key + (first_tile + t) * KT + MINE * half;
        const int seen = (live ? min(place, r.keys - 1) + 1 : place) - key0, hidden = first - key0;  // of these keys, from `hidden` on and before `seen`
        float tops[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        if (__all_sync(0xffffffffu, seen >= MINE && hidden <= 0)) {
#pragma unroll
          for (int j = 0; j < MINE; ++j) s[j] *= p.scale_log2, tops[j & 3] = fmaxf(tops[j & 3], s[j]);
        } else {
#pragma unroll
          for (int j = 0; j < MINE; ++j) s[j] = j < seen && j >= hidden ? s[j] * p.scale_log2 : -INFINITY, tops[j & 3] = fmaxf(tops[j & 3], s[j]);
        }
        top = fmaxf(fmaxf(tops[0], tops[1]), fmaxf(tops[2], tops[3]));
        if (row < L_ROWS) row_top[t & 1][half][row] = top;
      }
      const bool grown = top > m + L_SLACK;  // (from -infinity: anything at all)
      const bool any = softmax_any(grown);
      float corr = 1.f;
      if (row < nr) {
        top = fmaxf(top, row_top[t & 1][half ^ 1][row]);
        if (top > m + L_SLACK) corr = exp2_fast(m - top), m = top;
        const float at = m == -INFINITY ? 0.f : m;
        float sums[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < MINE; ++j) s[j] = exp2_fast(s[j] - at), sums[j & 3] += s[j];
        l = l * corr + ((sums[0] + sums[1]) + (sums[2] + sums[3]));
      }
      if (t > 0) {  // the sums and P are free once the last tile's MMAs are done
        mbar_wait(smem_u32(pv_done), (t - 1) & 1, abort_flag, LW_PV);
        tc_fence_after();
        if (any) {
          if (row < L_ROWS && half == 0) row_scale[row] = corr;
          softmax_sync();
          for (int i = half; i < p.blocks * (nr / 16); i += 2) {
            const int b = i / (nr / 16), c = i % (nr / 16) * 16;
            float v[16];
            tmem_ld16_nowait(tO + lanes + b * nr + c, v);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 16; ++e) v[e] *= row_scale[c + e];
            tmem_st16(tO + lanes + b * nr + c, v);
          }
          tmem_st_wait();
        }
      }
      if (row < nr) {
#pragma unroll
        for (int c = 0; c < MINE / 8; ++c)
          st_shared_v4(sP + row * 128 + (((MINE / 8 * half + c) ^ (row & 7)) << 4), pack_bf16x2(s[8 * c], s[8 * c + 1]), pack_bf16x2(s[8 * c + 2], s[8 * c + 3]),
                       pack_bf16x2(s[8 * c + 4], s[8 * c + 5]), pack_bf16x2(s[8 * c + 6], s[8 * c + 7]));
      }
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(p_full));
    }
    // ---- the result: through the ring's shared memory, from where the tile's rows - one piece of memory - leave in one copy
    if (n_tiles) {
      mbar_wait(smem_u32(pv_done), (n_tiles - 1) & 1, abort_flag, LW_PV);
      tc_fence_after();
    }
    if (row < L_ROWS && half == 1) row_top[0][1][row] = l;
    softmax_sync();
    const int64_t part = (int64_t)tile * p.splits + split;
    if (row < L_ROWS && half == 0) {
      l += row_top[0][1][row];
      float f = 1.f;
      if (p.clustered) {
        row_top[0][0][row] = m, row_top[1][0][row] = l;
      } else if (p.splits > 1) {
        p.part_ml[(part * L_ROWS + row) * 2] = m, p.part_ml[(part * L_ROWS + row) * 2 + 1] = l;
      } else {
        float total = l;
        if (a.sink && live) {
          const float sink = a.sink[(r.first_row + row) % a.heads] * 1.4426950408889634f, top = fmaxf(m, sink);
          f = exp2f(m - top), total = l * f + exp2f(sink - top);
        }
        f = total > 0.f ? f / total : 0.f;
      }
      row_scale[row] = f;
    }
    softmax_sync();
    if (n_tiles || p.splits == 1) {
      const uint32_t pitch = (uint32_t)a.rank * (p.splits > 1 ? 4 : 2);
#pragma unroll 1
      for (int i = half; i < p.blocks * (nr / 16); i += 2) {  // (short code: it runs once, and is fetched as it runs)
        const int b = i / (nr / 16), c = i % (nr / 16) * 16, d = 128 * b + row;
        float v[16];
        if (n_tiles) {
          tmem_ld16_nowait(tO + lanes + b * nr + c, v);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int e = 0; e < 16; ++e) v[e] = 0.f;
        }
        if (d >= a.rank) continue;
        uint32_t at = sK + c * pitch + d * (p.splits > 1 ? 4 : 2);
        if (p.splits > 1) {
#pragma unroll
          for (int e = 0; e < 16; ++e, at += pitch) asm volatile("st.shared.f32 [%0], %1;" ::"r"(at), "f"(v[e]) : "memory");
        } else {
#pragma unroll
          for (int e = 0; e < 16; ++e, at += pitch) asm volatile("st.shared.u16 [%0], %1;" ::"r"(at), "h"((uint16_t)float_to_bf16_bits(v[e] * row_scale[c + e])) : "memory");
        }
      }
      fence_proxy_async();
      softmax_sync();
      if (tid == 0 && !p.clustered) {
        if (p.splits > 1) bulk_copy_s2g(p.part_o + part * L_ROWS * a.rank, sK, (uint32_t)(r.rows * a.rank * 4));
        else bulk_copy_s2g(static_cast<uint16_t*>(a.out) + r.first_row * a.rank, sK, (uint32_t)(r.rows * a.rank * 2));
      }
    }
  }
  tc_fence_before();
  __syncwarp();
  if (p.clustered) {
    cluster_barrier();  // every CTA's part - sums, maxima, weights' totals - is in its shared memory
    if (warp < L_SOFTMAX / 32) {
      const int share = (r.rows + p.splits - 1) / p.splits, c0 = split * share, mine = max(0, min(r.rows, c0 + share) - c0);
      float* weight = reinterpret_cast<float*>(smem + (sP - sQ));  // [rows][8]
      // (the others' numbers are asked for all at once: four CTAs' at a time, the last one's again past the end)
      if (tid < mine) {
        const uint32_t top_at = smem_u32(&row_top[0][0][c0 + tid]), sum_at = smem_u32(&row_top[1][0][c0 + tid]);
        const float sink = a.sink ? a.sink[(r.first_row + c0 + tid) % a.heads] * 1.4426950408889634f : -INFINITY;
        float ms[8], ls[8], top = sink;
#pragma unroll
        for (int s0 = 0; s0 < 8; s0 += 4) {
#pragma unroll
          for (int s = s0; s < s0 + 4; ++s) ms[s] = -INFINITY, ls[s] = 0.f;
          if (s0 < p.splits) {
#pragma unroll
            for (int s = s0; s < s0 + 4; ++s) ms[s] = load_cluster_f32(top_at, min(s, p.splits - 1)), ls[s] = load_cluster_f32(sum_at, min(s, p.splits - 1));
          }
        }
#pragma unroll
        for (int s = 0; s < 8; ++s) {
          if (s >= p.splits) ms[s] = -INFINITY, ls[s] = 0.f;
          top = fmaxf(top, ms[s]);
        }
        const float at = top == -INFINITY ? 0.f : top;
        float total = exp2f(sink - at);
#pragma unroll
        for (int s = 0; s < 8; ++s) ms[s] = exp2_fast(ms[s] - at), total += ls[s] * ms[s];
#pragma unroll
        for (int s = 0; s < 8; ++s) weight[tid * 8 + s] = ls[s] > 0.f ? ms[s] / total : 0.f;
      }
      softmax_sync();
      // a warp takes pieces of 128 columns of a row, two at a time, every CTA's part of both on its way at once
      const int pieces = (a.rank + 127) / 128, all = mine * pieces;
#pragma unroll 1
      for (int i = 2 * warp; i < all; i += 2 * (L_SOFTMAX / 32)) {
        float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        int c[2], d[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int j = min(i + u, all - 1);
          c[u] = j / pieces, d[u] = min((j - c[u] * pieces) * 128 + 4 * lane, a.rank - 4);  // (rank is a multiple of 8)
        }
#pragma unroll 1
        for (int s0 = 0; s0 < p.splits; s0 += 4) {
          float v[2][4][4];
#pragma unroll
          for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int s = 0; s < 4; ++s) load_cluster_v4(sK + (uint32_t)((c0 + c[u]) * a.rank + d[u]) * 4, min(s0 + s, p.splits - 1), v[u][s]);
#pragma unroll
          for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int s = 0; s < 4; ++s) {
              const float f = weight[c[u] * 8 + s0 + s];  // (0 past the last CTA, and for one without keys, which left nothing there)
#pragma unroll
              for (int e = 0; e < 4; ++e) acc[u][e] += f > 0.f ? f * v[u][s][e] : 0.f;
            }
        }
#pragma unroll
        for (int u = 0; u < 2; ++u)
          if (i + u < all)
            *reinterpret_cast<uint2*>(static_cast<uint16_t*>(a.out) + (r.first_row + c0 + c[u]) * a.rank + d[u]) =
                make_uint2(pack_bf16x2(acc[u][0], acc[u][1]), pack_bf16x2(acc[u][2], acc[u][3]));
      }
    }
    cluster_barrier();  // the others have read this CTA's part
  }
  __syncthreads();
  if (warp == L_WARP_MMA) {
    tc_fence_after();
    tmem_dealloc(tmem, p.tmem_cols);
  }
}

// a block per (token, head): its splits' sums weighted by their maxima, the sink beside them
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentParams p) {
  griddep_launch_dependents();
  griddep_wait();
  const LatentArgs& a = p.a;
  const int64_t id = blockIdx.x;
  int64_t tile;
  int row;
  if (p.tiles_per_token) {
    const int h = (int)(id % a.heads);
    tile = id / a.heads * p.tiles_per_token + h / L_ROWS, row = h % L_ROWS;
  } else {
    tile = id / L_ROWS, row = (int)(id % L_ROWS);
  }
  const float* ml = p.part_ml + (tile * p.splits * L_ROWS + row) * 2;
  const float sink = a.sink ? a.sink[id % a.heads] * 1.4426950408889634f : -INFINITY;
  float m = sink;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ml[s * L_ROWS * 2]);
  const float at = m == -INFINITY ? 0.f : m;
  float total = exp2f(sink - at);
  for (int s = 0; s < p.splits; ++s) total += ml[s * L_ROWS * 2 + 1] * exp2f(ml[s * L_ROWS * 2] - at);
  const float inv = total > 0.f ? 1.f / total : 0.f;
  for (int d = threadIdx.x; d < a.rank; d += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < p.splits; ++s)
      if (ml[s * L_ROWS * 2 + 1] > 0.f) acc += p.part_o[((tile * p.splits + s) * L_ROWS + row) * a.rank + d] * exp2f(ml[s * L_ROWS * 2] - at);
    static_cast<uint16_t*>(a.out)[id * a.rank + d] = (uint16_t)float_to_bf16_bits(acc * inv);
  }
}

// sizes and launch shape; false: not for this kernel
bool make_latent_plan(int64_t T, int heads, int rank, int rot, int64_t max_keys, int chunk, int window, LatentParams& p) {
  if (window > 0) {  // (a tile of a chunk's pairs sees the windows of all its tokens)
    const int64_t most = window + (chunk ? ceil_div(L_ROWS, heads) : 0);
    max_keys = most < max_keys ? most : max_keys;
  }
  const int W = rank + rot;
  if (W % 8 || rank % 8 || W > 64 * L_MAX_CHUNKS || rank > 128 * L_MAX_BLOCKS || max_keys < 1) return false;
  const int64_t rows = chunk ? T * heads : heads;
  p.nr = rows >= L_ROWS ? L_ROWS : (int)ceil_div(rows, 16) * 16;
  p.chunks = (int)ceil_div(W, 64), p.blocks = (int)ceil_div(rank, 128);
  const size_t fixed = 1024 + (size_t)p.chunks * p.nr * 128 + L_ROWS * 128;
  for (p.keys = 64; p.keys >= 32; p.keys -= 16) {
    p.bufs = fixed < L_SMEM ? (int)((L_SMEM - fixed) / ((size_t)p.chunks * p.keys * 128)) : 0;
    if (p.bufs >= 3) break;
  }
  if (p.bufs < 3) return false;
  p.bufs = p.bufs > L_MAX_BUFS ? L_MAX_BUFS : p.bufs;
  // (an A operand reads 128 rows from a Q chunk's start, and two 64-column chunks from a cache tile's last: both stay within the ring and P)
  const int cols = 128 + p.blocks * p.nr;
  p.tmem_cols = 32;
  while (p.tmem_cols < cols) p.tmem_cols *= 2;
  if (p.tmem_cols > 512) return false;
  p.tiles_per_token = chunk ? 0 : (int)ceil_div(heads, L_ROWS);
  const int64_t tiles = chunk ? ceil_div(rows, L_ROWS) : T * p.tiles_per_token;
  if (tiles > (1 << 20)) return false;
  const int sms = sm_count_of_device();
  const int64_t key_tiles = ceil_div(max_keys, p.keys);
  int best = 1;
  double best_cost = 1e30;
  for (int s = 1; s <= 32 && s <= key_tiles; ++s) {  // tiles of keys a CTA, plus its fixed cost in the same unit, by rounds of CTAs
    if ((s > 1 && s < 8 && tiles * s > sms - s) || (s == 8 && tiles * s > 128)) continue;  // (a cluster's CTAs run together: one round of them)
    const double cost = (double)ceil_div(tiles * s, sms) * ((double)ceil_div(key_tiles, s) + 3.0) + (s > 8 ? 4.0 + 0.05 * s : s > 1 ? 1.0 : 0.0);
    if (cost < best_cost - 1e-9) best_cost = cost, best = s;
  }
  p.splits = best, p.clustered = best > 1 && best <= 8;
  return true;
}

int64_t latent_tiles(const LatentParams& p, int64_t T, int heads) { return p.tiles_per_token ? T * p.tiles_per_token : ceil_div(T * heads, L_ROWS); }

}  // namespace

size_t latent_tcgen05_workspace(int64_t T, int heads, int rank, int rot, int64_t max_keys, int chunk, int window) {
  LatentParams p{};
  if (T < 1 || !make_latent_plan(T, heads, rank, rot, max_keys, chunk, window, p) || p.splits == 1 || p.clustered) return 0;
  return (size_t)latent_tiles(p, T, heads) * p.splits * L_ROWS * (rank + 2) * sizeof(float);
}

bool latent_tcgen05_supports(const LatentArgs& a) {
  LatentParams p{};
  return tma_encoder() != nullptr && a.ld_q == (int64_t)a.heads * (a.rank + a.rot) && a.ld_o == (int64_t)a.heads * a.rank && (uintptr_t)a.q % 16 == 0 &&
         (uintptr_t)a.cache % 16 == 0 && (uintptr_t)a.out % 16 == 0 && a.cache_rows < (1ll << 31) && a.T * a.heads < (1ll << 31) && make_latent_plan(a.T, a.heads, a.rank, a.rot, a.max_keys, a.chunk, a.window, p);
}

int latent_tcgen05(const LatentArgs& a, cudaStream_t s) {
  LatentParams p{};
  p.a = a;
  make_latent_plan(a.T, a.heads, a.rank, a.rot, a.max_keys, a.chunk, a.window, p);
  p.scale_log2 = a.scale * 1.4426950408889634f;
  const int64_t tiles = latent_tiles(p, a.T, a.heads);
  if (p.splits > 1 && !p.clustered) {
    const size_t need = latent_tcgen05_workspace(a.T, a.heads, a.rank, a.rot, a.max_keys, a.chunk, a.window);
    if (!a.workspace || a.workspace_bytes < need) {
      set_error("fb_latent_attention: workspace of %zu bytes needed, %zu given", need, a.workspace_bytes);
      return FB_ERR_MEMORY;
    }
    p.part_o = (float*)a.workspace, p.part_ml = p.part_o + (size_t)tiles * p.splits * L_ROWS * a.rank;
  }
  const int W = a.rank + a.rot;
  LatentMaps maps{};
  const int64_t strides[2] = {W, 64};
  const int whole = W / 64;
  for (int which = 0; which < 2; ++which) {
    const void* base = which ? a.cache : a.q;
    const int64_t rows = which ? a.cache_rows : a.T * a.heads;
    const int box = which ? p.keys : p.nr;
    if (whole) {
      const int64_t d[3] = {64, rows, whole};
      const int b[3] = {64, box, whole};
      if (int rc = tma_map_bf16(which ? &maps.k : &maps.q, base, 3, d, strides, b, "fb_latent_attention")) return rc;
    }
    if (whole < p.chunks) {
      const int64_t d[2] = {W, rows};
      const int b[2] = {64, box};
      if (int rc = tma_map_bf16(which ? &maps.k_tail : &maps.q_tail, base, 2, d, strides, b, "fb_latent_attention")) return rc;
    }
  }
  const auto kernel = p.keys == 64 ? latent_tcgen05_kernel<64> : p.keys == 48 ? latent_tcgen05_kernel<48> : latent_tcgen05_kernel<32>;
  static std::atomic<uint64_t> opted[3];
  if (first_on_device(opted[p.keys / 16 - 2])) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)L_SMEM);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3((unsigned)tiles, (unsigned)p.splits), cfg.blockDim = dim3(L_THREADS), cfg.stream = s;
  cfg.dynamicSmemBytes = 1024 + (size_t)p.chunks * p.nr * 128 + (size_t)p.bufs * p.chunks * p.keys * 128 + L_ROWS * 128;
  // (room for what an A operand reads past Q's last rows where the ring is short)
  const size_t reach = 1024 + (size_t)(p.chunks - 1) * p.nr * 128 + 128 * 128;
  if (cfg.dynamicSmemBytes < reach) cfg.dynamicSmemBytes = reach;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = 1, attr[1].val.clusterDim.y = (unsigned)p.splits, attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr, cfg.numAttrs = p.clustered ? 2 : 1;
  cudaLaunchKernelEx(&cfg, kernel, maps, p);
  if (p.splits > 1 && !p.clustered) {
    cfg.numAttrs = 1;
    cfg.gridDim = dim3((unsigned)(a.T * a.heads)), cfg.blockDim = dim3(128), cfg.dynamicSmemBytes = 0;
    cudaLaunchKernelEx(&cfg, latent_combine_kernel, p);
  }
  return launch_status("fb_latent_attention");
}

static const StatusWord g_status_reader(read_and_clear_status_word);

}  // namespace fb
