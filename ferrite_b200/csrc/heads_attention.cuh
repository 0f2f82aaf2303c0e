// The tensor-core kernel of fb_heads_attention (heads_attention.cu says how it works), and its launch for keys of one width; a
// source file a width instantiates it, so that they compile side by side.
#pragma once
#include "heads.cuh"
#include "launch.cuh"
#include "mma_sync.cuh"
#include "sm100.cuh"
#include "tma_host.cuh"

namespace fb {

constexpr int HA_KEYS = 64, HA_MAX_STAGES = 6;
enum HeadsWait { HW_EMPTY = 601, HW_FULL };
constexpr float LOG2E = 1.4426950408889634f;

template <int THREADS>
__device__ __forceinline__ void consumers_sync() { asm volatile("barrier.cta.sync.aligned 1, %0;" ::"n"(THREADS) : "memory"); }

// a tile's form: WR warps by rows (each MT tiles of 16), WK by keys; one more warp asks for the tiles
template <int DK, int DV, int WR, int WK, int MT>
struct HeadsShape {
  static constexpr int ROWS = 16 * WR * MT, QP = DK * 2 + 16;                                // row pitch of the queries: an odd number of 16-byte pieces
  static constexpr int CHUNK = HA_KEYS * 128, STAGE = (DK + DV) / 64 * CHUNK;                // 64 columns of a tile's keys or values, in 128-byte swizzled rows
  static constexpr int ML = WK * ROWS * DV * 4, PARTS = ML + WK * ROWS * 8;                  // after the loop: the warps' sums, maxima and denominators
  static constexpr int Q = ROWS * QP;
  // (the ring is first, then the queries)
  static constexpr int smem(int stages) { return 1024 + (stages * STAGE > PARTS ? stages * STAGE : PARTS) + Q; }
};

template <int DK, int DV, int WR, int WK, int MT>
__global__ void __launch_bounds__(32 * WR * WK + 32) heads_attention_kernel(const __grid_constant__ CUtensorMap map, const HeadsArgs a) {
  using S = HeadsShape<DK, DV, WR, WK, MT>;
  constexpr int THREADS = 32 * WR * WK, ROWS = S::ROWS, NT = HA_KEYS / WK / 8;  // NT: 8-key tiles of a warp
  constexpr bool KEEP_Q = MT * DK <= 128;
  griddep_launch_dependents();
  extern __shared__ uint8_t heads_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(heads_smem) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem + (a.stages * S::STAGE > S::PARTS ? a.stages * S::STAGE : S::PARTS);
  __shared__ uint64_t full[HA_MAX_STAGES], empty[HA_MAX_STAGES];
  __shared__ uint32_t abort_word;
  const uint32_t abort_flag = smem_u32(&abort_word);
  const int tid = threadIdx.x, warp = uniform_warp(), lane = tid & 31, wr = warp / WK, wk = warp % WK;
  if (tid == 0) {
    for (int i = 0; i < a.stages; ++i) mbar_init(smem_u32(full + i), 1), mbar_init(smem_u32(empty + i), WR * WK);
    abort_word = 0;
    fence_barrier_init();
  }
  __syncthreads();
  const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y;
  const int entry = blockIdx.z / a.tiles, tile = a.tiles - 1 - blockIdx.z % a.tiles;  // (a chunk's last tiles see the most keys: they start first)
  const int pair0 = tile * ROWS, rows = min(ROWS, a.pairs - pair0);
  const int64_t token0 = a.chunk ? 0 : entry;
  griddep_wait();

  // the keys this tile's pairs see, cut into `splits` runs
  const int tok_a = pair0 / a.rep, tok_b = (pair0 + rows - 1) / a.rep;
  int len = 0, lo = 0x7fffffff;
  for (int t = tok_a + lane; t <= tok_b; t += 32) {
    const int p = a.last[token0 + t];
    len = max(len, p + 1), lo = min(lo, first_seen(a, p));
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) len = max(len, __shfl_xor_sync(0xffffffffu, len, o)), lo = min(lo, __shfl_xor_sync(0xffffffffu, lo, o));
  const int64_t seq = (a.base ? a.base[token0] : 0) + a.row0;
  const int64_t room = seq < 0 ? 0 : a.cache_rows - seq;  // no key outside the cache is read
  len = (int)max((int64_t)0, min((int64_t)len, room));
  lo = max(0, min(lo, len));
  const int per = (len - lo + splits * HA_KEYS - 1) / (splits * HA_KEYS) * HA_KEYS;
  const int k0 = lo + split * per, k1 = min(len, k0 + per), n_tiles = k1 > k0 ? (k1 - k0 + HA_KEYS - 1) / HA_KEYS : 0;
  if (warp == WR * WK) {  // the tiles: keys, then values, 64 columns a copy
    if (lane == 0) {
      int slot = 0, i = 0;
      uint32_t phase = 0;
      bool ok = true;
      const int ck = (a.dim + 63) / 64, cv = (a.vdim + 63) / 64;
      for (; i < n_tiles; ++i) {
        ok = mbar_wait(smem_u32(empty + slot), phase ^ 1, abort_flag, HW_EMPTY);
        if (!ok) break;
        const uint32_t bar = smem_u32(full + slot), to = smem_u32(smem) + slot * S::STAGE;
        mbar_expect_tx(bar, (uint32_t)(ck + cv) * S::CHUNK);
        for (int c = 0; c < ck; ++c) tma_load_3d(to + c * S::CHUNK, &map, 64 * c, (int)seq + k0 + i * HA_KEYS, g, bar);
        for (int c = 0; c < cv; ++c) tma_load_3d(to + (DK / 64 + c) * S::CHUNK, &map, a.dim + 64 * c, (int)seq + k0 + i * HA_KEYS, g, bar);
        if (++slot == a.stages) slot = 0, phase ^= 1;
      }
      if (!ok)  // given up: the copies under way land before this CTA's shared memory is anyone else's
        for (int b = 0; b < a.stages && b < i; ++b) {
          const long long start = clock64();
          while (!mbar_try_wait(smem_u32(full + b), b < slot ? phase : phase ^ 1) && clock64() - start < WAIT_CLOCKS) {
          }
        }
    }
    __syncwarp();
    if (splits == 1) return;
    cluster_barrier(), cluster_barrier();
    return;
  }

  int place_r[MT][2], lo_r[MT][2];  // this lane's rows: 16 (WR mt + wr) + lane / 4 and that + 8
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = 16 * (WR * mt + wr) + (lane >> 2) + 8 * h;
      place_r[mt][h] = r < rows ? a.last[token0 + (pair0 + r) / a.rep] : -1;
      lo_r[mt][h] = r < rows ? first_seen(a, place_r[mt][h]) : 0;
    }
  // the queries; past a key's columns zeros, so that what a tile holds there (its values' first) does not count
  for (int c = tid; c < ROWS * (DK / 8); c += THREADS) {
    const int r = c / (DK / 8), ch = c % (DK / 8), pair = pair0 + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < rows && ch < a.dim / 8)
      v = *reinterpret_cast<const uint4*>(static_cast<const uint16_t*>(a.q) + (token0 + pair / a.rep) * a.ld_q + ((int64_t)g * a.rep + pair % a.rep) * a.dim + ch * 8);
    *reinterpret_cast<uint4*>(sQ + r * S::QP + ch * 16) = v;
  }
  consumers_sync<THREADS>();
  const int mi = lane >> 3, ml = lane & 7;
  const uint32_t q_at = smem_addr(sQ) + (16 * wr + (mi & 1) * 8 + ml) * S::QP + (mi >> 1) * 16;
  uint32_t qf[KEEP_Q ? DK / 16 : 1][MT][4];
  if constexpr (KEEP_Q) {
#pragma unroll
    for (int kt = 0; kt < DK / 16; ++kt)
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) ldmatrix_x4(q_at + mt * 16 * WR * S::QP + kt * 32, qf[kt][mt]);
  }

  float o[MT][DV / 8][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;
  float m_run[MT][2], l_run[MT][2];  // maxima of the unscaled scores
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) m_run[mt][0] = m_run[mt][1] = -INFINITY, l_run[mt][0] = l_run[mt][1] = 0.f;
  const float scale_log2 = a.scale * LOG2E;
  const SoftCap cap = soft_cap(a);
  float bias_r[MT][2];  // weights by sigmoid: the rows' numbers; such parts have the maximum 0 and are added up as they are
  if (a.key_bias) {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = 16 * (WR * mt + wr) + (lane >> 2) + 8 * h;
        bias_r[mt][h] = r < rows ? a.key_bias[g * a.rep + (pair0 + r) % a.rep] * LOG2E : 0.f, m_run[mt][h] = 0.f;
      }
  }

  // where a lane's 16 bytes stand within a swizzled row, for the four steps of 16 columns that a row has
  uint32_t k_off[4], v_off[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) k_off[j] = ((2 * j + (mi & 1)) ^ ml) << 4, v_off[j] = ((2 * j + (mi >> 1)) ^ ml) << 4;
  int slot = 0;
  uint32_t phase = 0;
  for (int i = 0; i < n_tiles; ++i) {
    mbar_wait(smem_u32(full + slot), phase, abort_flag, HW_FULL);
    const int krow = (HA_KEYS / WK) * wk;
    const uint32_t kb = smem_addr(smem) + slot * S::STAGE + (krow + (mi >> 1) * 8 + ml) * 128;
    const uint32_t vb = smem_addr(smem) + slot * S::STAGE + DK / 64 * S::CHUNK + (krow + (mi & 1) * 8 + ml) * 128;
    float s[MT][NT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int n = 0; n < NT; ++n) s[mt][n][0] = s[mt][n][1] = s[mt][n][2] = s[mt][n][3] = 0.f;
#pragma unroll
    for (int kt = 0; kt < DK / 16; ++kt) {
      uint32_t qk[MT][4];
      if constexpr (!KEEP_Q) {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) ldmatrix_x4(q_at + mt * 16 * WR * S::QP + kt * 32, qk[mt]);
      }
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        uint32_t b[4];
        ldmatrix_x4(kb + n * 8 * 128 + (kt >> 2) * S::CHUNK + k_off[kt & 3], b);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(s[mt][n], KEEP_Q ? qf[KEEP_Q ? kt : 0][mt] : qk[mt], b[0], b[1]);
          mma_bf16(s[mt][n + 1], KEEP_Q ? qf[KEEP_Q ? kt : 0][mt] : qk[mt], b[2], b[3]);
        }
      }
    }
    const int key0 = k0 + i * HA_KEYS + krow, key_first = key0 + (lane & 3) * 2, key_end = key0 + HA_KEYS / WK;
    uint32_t pf[MT][NT / 2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      if (cap.in > 0.f) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[mt][n][e] = capped(cap, s[mt][n][e]);
      }
      // (a whole tile that every pair of the warp sees needs no mask)
      if (!__all_sync(0xffffffffu, key_end <= k1 && min(place_r[mt][0], place_r[mt][1]) >= key_end - 1 && max(lo_r[mt][0], lo_r[mt][1]) <= key0)) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int key = key_first + n * 8 + (e & 1);
            if (key >= k1 || key > place_r[mt][e >> 1] || key < lo_r[mt][e >> 1]) s[mt][n][e] = -INFINITY;
          }
      }
      if (a.key_bias) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            float x, y;
            sigmoid_pair(fmaf(s[mt][n][2 * h], scale_log2, bias_r[mt][h]), fmaf(s[mt][n][2 * h + 1], scale_log2, bias_r[mt][h]), x, y);
            pf[mt][n / 2][2 * (n & 1) + h] = pack_bf16x2(s[mt][n][2 * h] == -INFINITY ? 0.f : x, s[mt][n][2 * h + 1] == -INFINITY ? 0.f : y);
          }
        continue;
      }
      float mx[2] = {m_run[mt][0], m_run[mt][1]}, corr[2];
#pragma unroll
      for (int n = 0; n < NT; ++n) mx[0] = fmaxf(mx[0], fmaxf(s[mt][n][0], s[mt][n][1])), mx[1] = fmaxf(mx[1], fmaxf(s[mt][n][2], s[mt][n][3]));
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
        const float safe = mx[h] == -INFINITY ? 0.f : mx[h];
        corr[h] = exp2_of((m_run[mt][h] - safe) * scale_log2);
        m_run[mt][h] = mx[h], l_run[mt][h] *= corr[h], mx[h] = -safe * scale_log2;
      }
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const float p0 = exp2_of(fmaf(s[mt][n][0], scale_log2, mx[0])), p1 = exp2_of(fmaf(s[mt][n][1], scale_log2, mx[0]));
        const float p2 = exp2_of(fmaf(s[mt][n][2], scale_log2, mx[1])), p3 = exp2_of(fmaf(s[mt][n][3], scale_log2, mx[1]));
        l_run[mt][0] += p0 + p1, l_run[mt][1] += p2 + p3;
        pf[mt][n / 2][2 * (n & 1)] = pack_bf16x2(p0, p1), pf[mt][n / 2][2 * (n & 1) + 1] = pack_bf16x2(p2, p3);
      }
      if (!__all_sync(0xffffffffu, corr[0] == 1.f && corr[1] == 1.f)) {
#pragma unroll
        for (int d = 0; d < DV / 8; ++d) o[mt][d][0] *= corr[0], o[mt][d][1] *= corr[0], o[mt][d][2] *= corr[1], o[mt][d][3] *= corr[1];
      }
    }
#pragma unroll
    for (int n = 0; n < NT / 2; ++n)
#pragma unroll
      for (int d = 0; d < DV / 8; d += 2) {
        uint32_t b[4];
        ldmatrix_x4_trans(vb + n * 16 * 128 + (d >> 3) * S::CHUNK + v_off[(d >> 1) & 3], b);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) mma_bf16(o[mt][d], pf[mt][n], b[0], b[1]), mma_bf16(o[mt][d + 1], pf[mt][n], b[2], b[3]);
      }
    __syncwarp();
    if (lane == 0) mbar_arrive(smem_u32(empty + slot));
    if (++slot == a.stages) slot = 0, phase ^= 1;
  }

#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      l_run[mt][h] += __shfl_xor_sync(0xffffffffu, l_run[mt][h], 1);
      l_run[mt][h] += __shfl_xor_sync(0xffffffffu, l_run[mt][h], 2);
      m_run[mt][h] *= scale_log2;
    }
  if (WK == 1 && splits == 1) {  // each row is one warp's: out of the registers
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = 16 * (WR * mt + wr) + (lane >> 2) + 8 * h;
        if (r >= rows) continue;
        const int pair = pair0 + r, head = g * a.rep + pair % a.rep;
        const int64_t t = token0 + pair / a.rep, col0 = (int64_t)head * a.vdim + (lane & 3) * 2;
        float m = m_run[mt][h], l = l_run[mt][h], f = 1.f;
        if (a.sink) {
          const float sink = a.sink[head] * LOG2E;
          m = fmaxf(m, sink), f = exp2_of(m_run[mt][h] - m), l = l * f + exp2_of(sink - m);
        }
        f = a.key_bias ? a.out_scale : l > 0.f ? f * a.out_scale / l : 0.f;
        uint16_t* out = static_cast<uint16_t*>(a.out) + t * a.ld_o;
#pragma unroll
        for (int d = 0; d < DV / 8; ++d)
          if (d * 8 < a.vdim)
            *reinterpret_cast<uint32_t*>(out + col0 + d * 8) = pack_bf16x2(o[mt][d][2 * h] * f * gate_of(a, t, col0 + d * 8), o[mt][d][2 * h + 1] * f * gate_of(a, t, col0 + d * 8 + 1));
      }
    return;
  }

  // each warp's sums, maxima and denominators to shared memory; then one owner a (row, column) over the warps and the cluster
  consumers_sync<THREADS>();  // (no warp reads the ring any more)
  float *so = reinterpret_cast<float*>(smem), *sml = reinterpret_cast<float*>(smem + S::ML);  // [WK][ROWS]
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    const int part = wk * ROWS + 16 * (WR * mt + wr) + (lane >> 2);
#pragma unroll
    for (int d = 0; d < DV / 8; ++d) {
      const int col = d * 8 + (lane & 3) * 2;
      if (col >= a.vdim) break;
      *reinterpret_cast<float2*>(so + part * DV + col) = make_float2(o[mt][d][0], o[mt][d][1]);
      *reinterpret_cast<float2*>(so + (part + 8) * DV + col) = make_float2(o[mt][d][2], o[mt][d][3]);
    }
    if ((lane & 3) == 0)
      sml[part * 2] = m_run[mt][0], sml[part * 2 + 1] = l_run[mt][0], sml[(part + 8) * 2] = m_run[mt][1], sml[(part + 8) * 2 + 1] = l_run[mt][1];
  }
  consumers_sync<THREADS>();
  if (WK > 1 && splits > 1) {  // the CTA's warps into one part, in place
    for (int idx = tid; idx < rows * a.vdim; idx += THREADS) {
      const int r = idx / a.vdim, d = idx % a.vdim;
      float m = -INFINITY, acc = 0.f;
#pragma unroll
      for (int w = 0; w < WK; ++w) m = fmaxf(m, sml[(w * ROWS + r) * 2]);
      m = m == -INFINITY ? 0.f : m;
#pragma unroll
      for (int w = 0; w < WK; ++w) acc += so[(w * ROWS + r) * DV + d] * exp2_of(sml[(w * ROWS + r) * 2] - m);
      so[r * DV + d] = acc;
    }
    consumers_sync<THREADS>();
    float mm = -INFINITY, ll = 0.f;
    if (tid < rows) {
#pragma unroll
      for (int w = 0; w < WK; ++w) mm = fmaxf(mm, sml[(w * ROWS + tid) * 2]);
      const float m = mm == -INFINITY ? 0.f : mm;
#pragma unroll
      for (int w = 0; w < WK; ++w) ll += sml[(w * ROWS + tid) * 2 + 1] * exp2_of(sml[(w * ROWS + tid) * 2] - m);
      sml[tid * 2] = mm, sml[tid * 2 + 1] = ll;
    }
    consumers_sync<THREADS>();
  }
  if (splits > 1) cluster_barrier();
  const int parts = splits > 1 ? splits : WK;
  for (int idx = splits > 1 ? split * THREADS + tid : tid; idx < rows * a.vdim; idx += splits > 1 ? splits * THREADS : THREADS) {
    const int r = idx / a.vdim, d = idx % a.vdim, pair = pair0 + r, head = g * a.rep + pair % a.rep;
    const int64_t t = token0 + pair / a.rep, col = (int64_t)head * a.vdim + d;
    float pm[8], pl[8], po[8];  // (all on their way before the first is needed)
    const float gate = gate_of(a, t, col);
#pragma unroll
    for (int p = 0; p < 8; ++p) {
      pm[p] = -INFINITY, pl[p] = po[p] = 0.f;
      if (p < parts) {
        if (splits > 1) {
          const uint32_t at = smem_addr(sml + r * 2);
          pm[p] = load_cluster_f32(at, p), pl[p] = load_cluster_f32(at + 4, p), po[p] = load_cluster_f32(smem_addr(so + r * DV + d), p);
        } else {
          pm[p] = sml[(p * ROWS + r) * 2], pl[p] = sml[(p * ROWS + r) * 2 + 1], po[p] = so[(p * ROWS + r) * DV + d];
        }
      }
    }
    float m = a.sink ? a.sink[head] * LOG2E : -INFINITY, l = 0.f, acc = 0.f;
    const float sink = m;
#pragma unroll
    for (int p = 0; p < 8; ++p) m = fmaxf(m, pm[p]);
    m = m == -INFINITY ? 0.f : m;
    if (a.sink) l = exp2_of(sink - m);
#pragma unroll
    for (int p = 0; p < 8; ++p) {
      const float f = exp2_of(pm[p] - m);
      l = fmaf(pl[p], f, l), acc = fmaf(po[p], f, acc);
    }
    static_cast<uint16_t*>(a.out)[t * a.ld_o + col] = (uint16_t)float_to_bf16_bits(a.key_bias ? acc * a.out_scale * gate : l > 0.f ? acc / l * a.out_scale * gate : 0.f);
  }
  if (splits > 1) cluster_barrier();  // the others have read this CTA's part
}

template <int DK, int DV, int WR, int WK, int MT>
static int launch_heads(HeadsArgs a, cudaStream_t s) {
  using S = HeadsShape<DK, DV, WR, WK, MT>;
  a.entries = a.chunk ? 1 : (int)a.T, a.pairs = a.chunk ? (int)a.T * a.rep : a.rep, a.tiles = (int)ceil_div(a.pairs, S::ROWS);
  // the keys over a cluster's CTAs where that makes for a shorter run of tiles: two CTAs an SM at a time, each with its own start and end
  const int64_t ctas = (int64_t)a.kv_heads * a.entries * a.tiles, key_tiles = ceil_div(a.seen, HA_KEYS);
  int splits = 1;
  for (int s = 2, best = (int)(ceil_div(ctas, 2 * 148) * (key_tiles + 2)); s <= 8 && key_tiles >= 2 * s; s *= 2) {
    const int64_t cost = ceil_div(ctas * s, 2 * 148) * (ceil_div(key_tiles, s) + 3);
    if (cost < best) best = (int)cost, splits = s;
  }
  // as many tiles in the ring as two CTAs an SM have room for, else one CTA's
  a.stages = HA_MAX_STAGES;
  while (a.stages > 3 && S::smem(a.stages) > 112 * 1024) --a.stages;
  if (S::smem(a.stages) > 112 * 1024 && S::smem(2) <= 112 * 1024) a.stages = 2;
  while (a.stages > 2 && S::smem(a.stages) > 225 * 1024) --a.stages;
  const int smem = S::smem(a.stages);
  CUtensorMap map;
  const int64_t dims[3] = {a.dim + a.vdim, a.cache_rows, a.kv_heads}, strides[2] = {a.dim + a.vdim, a.head_stride};
  const int box[3] = {64, HA_KEYS, 1};
  if (int rc = tma_map_bf16(&map, a.cache, 3, dims, strides, box, "fb_heads_attention (cache)")) return rc;
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(heads_attention_kernel<DK, DV, WR, WK, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3((unsigned)splits, (unsigned)a.kv_heads, (unsigned)(a.entries * a.tiles)), cfg.blockDim = dim3(32 * WR * WK + 32);
  cfg.dynamicSmemBytes = smem, cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = (unsigned)splits, attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr, cfg.numAttrs = splits > 1 ? 2 : 1;
  cudaLaunchKernelEx(&cfg, heads_attention_kernel<DK, DV, WR, WK, MT>, map, a);
  return launch_status("fb_heads_attention");
}

template <int DK, int DV>
static int launch_form(const HeadsArgs& a, cudaStream_t s) {
  return a.chunk ? launch_heads<DK, DV, 4, 1, (DV <= 128 ? 2 : 1)>(a, s) : launch_heads<DK, DV, 1, 4, 1>(a, s);
}

template <int DK>
static int launch_values(const HeadsArgs& a, cudaStream_t s) {
  return a.vdim <= 64 ? launch_form<DK, 64>(a, s) : a.vdim <= 128 ? launch_form<DK, 128>(a, s) : launch_form<DK, 256>(a, s);
}

static const StatusWord g_status_reader(read_and_clear_status_word);

}  // namespace fb
