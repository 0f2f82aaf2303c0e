// Attention with grouped key heads over a cache whose rows are a key and then its value: the two may differ in width, the
// keys a token sees may be confined to its own span of the sequence (spans of `span` places, counted from its start), a
// number per head may join the softmax's denominator, and the output may be gated column by column.
//
// A CTA has one key head, a tile of (token, query head) pairs that share it - the pairs of one token in a decode step, those
// of consecutive tokens in a prompt's chunk - and a run of the keys that they see; 64-key tiles come in by cp.async, double
// buffered; q k^T and p v run on mma.sync with an online softmax in registers.
//   prompt   128 pairs (values of more than 128 columns: 64), a warp 32 of them over all keys of a tile
//   decode   16 pairs, a warp a quarter of a tile's keys; merged in shared memory
// The runs of one tile's keys are a cluster's CTAs: their parts are merged over distributed shared memory, so no result
// passes through global memory and there is no second kernel.
//
// bf16 rows of whole 16-byte pieces, heads of up to 256 columns; everything else (fp32, odd or wider heads) takes a plain
// kernel at the end of the file.
#include "heads.cuh"
#include "launch.cuh"
#include "mma_sync.cuh"
#include "sm100.cuh"

namespace fb {

constexpr int HA_KEYS = 64;
constexpr float LOG2E = 1.4426950408889634f;

// a tile's form: WR warps by rows (each MT tiles of 16), WK by keys
template <int DK, int DV, int WR, int WK, int MT>
struct HeadsShape {
  static constexpr int ROWS = 16 * WR * MT, QP = DK * 2 + 16, VP = DV * 2 + 16;  // row pitches in bytes: an odd number of 16-byte pieces
  static constexpr int Q = 0, K = ROWS * QP, V = K + 2 * HA_KEYS * QP, END = V + 2 * HA_KEYS * VP;
  static constexpr int O = 0, ML = O + WK * ROWS * DV * 4, PARTS = ML + WK * ROWS * 8;  // after the loop: the warps' sums, maxima and denominators
  static constexpr int SMEM = END > PARTS ? END : PARTS;
};

template <int DK, int DV, int WR, int WK, int MT>
__global__ void __launch_bounds__(32 * WR * WK) heads_attention_kernel(const HeadsArgs a) {
  using S = HeadsShape<DK, DV, WR, WK, MT>;
  constexpr int THREADS = 32 * WR * WK, ROWS = S::ROWS, NT = HA_KEYS / WK / 8;  // NT: 8-key tiles of a warp
  constexpr bool KEEP_Q = MT * DK <= 128;
  griddep_launch_dependents();
  extern __shared__ __align__(128) uint8_t heads_smem[];
  uint8_t* smem = heads_smem;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wr = warp / WK, wk = warp % WK;
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
    len = max(len, p + 1), lo = min(lo, span_start(p, a.span));
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) len = max(len, __shfl_xor_sync(0xffffffffu, len, o)), lo = min(lo, __shfl_xor_sync(0xffffffffu, lo, o));
  const int64_t seq = (a.base ? a.base[token0] : 0) + a.row0;
  const int64_t room = seq < 0 ? 0 : a.cache_rows - seq;  // no key outside the cache is read
  len = (int)max((int64_t)0, min((int64_t)len, room));
  lo = max(0, min(lo, len));
  const int per = (len - lo + splits * HA_KEYS - 1) / (splits * HA_KEYS) * HA_KEYS;
  const int k0 = lo + split * per, k1 = min(len, k0 + per), n_tiles = k1 > k0 ? (k1 - k0 + HA_KEYS - 1) / HA_KEYS : 0;
  const int W = a.dim + a.vdim;
  const uint16_t* cache = static_cast<const uint16_t*>(a.cache) + g * a.head_stride + (len > 0 ? (seq + k0) * W : 0);
  int place_r[MT][2], lo_r[MT][2];  // this lane's rows: 16 (WR mt + wr) + lane / 4 and that + 8
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = 16 * (WR * mt + wr) + (lane >> 2) + 8 * h;
      place_r[mt][h] = r < rows ? a.last[token0 + (pair0 + r) / a.rep] : -1;
      lo_r[mt][h] = r < rows ? span_start(place_r[mt][h], a.span) : 0;
    }

  // a thread's 16-byte pieces of a tile: piece tid, tid + THREADS, ... of 64 rows of a key's pieces and its value's
  const int kc = a.dim / 8, wc = W / 8, r_step = THREADS / wc, c_step = THREADS % wc, r_first = tid / wc, c_first = tid % wc;
  auto load_tile = [&](int i) {
    const uint32_t sk = smem_addr(smem + S::K + (i & 1) * HA_KEYS * S::QP), sv = smem_addr(smem + S::V + (i & 1) * HA_KEYS * S::VP);
    const int key0 = i * HA_KEYS, most = k1 - k0 - 1;
    // (rows past the end repeat the last key: their scores are masked, and their values are numbers)
    for (int r = r_first, c = c_first; r < HA_KEYS;) {
      const uint16_t* src = cache + (int64_t)min(key0 + r, most) * W + c * 8;
      cp_async16(c < kc ? sk + r * S::QP + c * 16 : sv + r * S::VP + (c - kc) * 16, src);
      r += r_step, c += c_step;
      if (c >= wc) c -= wc, ++r;
    }
    cp_async_commit();
  };
  if (n_tiles) load_tile(0);
  if (kc < DK / 8)  // a key is narrower than its room: the rest is zeros, in both buffers
    for (int c = tid; c < 2 * HA_KEYS * (DK / 8); c += THREADS) {
      const int r = c / (DK / 8), ch = c % (DK / 8);
      if (ch >= kc) *reinterpret_cast<uint4*>(smem + S::K + r * S::QP + ch * 16) = make_uint4(0, 0, 0, 0);
    }
  for (int c = tid; c < ROWS * (DK / 8); c += THREADS) {
    const int r = c / (DK / 8), ch = c % (DK / 8), pair = pair0 + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < rows && ch < kc)
      v = *reinterpret_cast<const uint4*>(static_cast<const uint16_t*>(a.q) + (token0 + pair / a.rep) * a.ld_q + ((int64_t)g * a.rep + pair % a.rep) * a.dim + ch * 8);
    *reinterpret_cast<uint4*>(smem + S::Q + r * S::QP + ch * 16) = v;
  }
  __syncthreads();
  const int mi = lane >> 3, ml = lane & 7;
  const uint32_t q_at = smem_addr(smem + S::Q) + (16 * wr + (mi & 1) * 8 + ml) * S::QP + (mi >> 1) * 16;
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

  for (int i = 0; i < n_tiles; ++i) {
    if (i + 1 < n_tiles) load_tile(i + 1);
    if (i + 1 < n_tiles) cp_async_wait<1>(); else cp_async_wait<0>();
    __syncthreads();
    const int krow = (HA_KEYS / WK) * wk;
    const uint32_t kb = smem_addr(smem + S::K + (i & 1) * HA_KEYS * S::QP) + (krow + (mi >> 1) * 8 + ml) * S::QP + (mi & 1) * 16;
    const uint32_t vb = smem_addr(smem + S::V + (i & 1) * HA_KEYS * S::VP) + (krow + (mi & 1) * 8 + ml) * S::VP + (mi >> 1) * 16;
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
        ldmatrix_x4(kb + n * 8 * S::QP + kt * 32, b);
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
        ldmatrix_x4_trans(vb + n * 16 * S::VP + d * 16, b);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) mma_bf16(o[mt][d], pf[mt][n], b[0], b[1]), mma_bf16(o[mt][d + 1], pf[mt][n], b[2], b[3]);
      }
    __syncthreads();  // the buffer is free for the tile after next
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
        f = l > 0.f ? f / l : 0.f;
        uint16_t* out = static_cast<uint16_t*>(a.out) + t * a.ld_o;
#pragma unroll
        for (int d = 0; d < DV / 8; ++d)
          if (d * 8 < a.vdim)
            *reinterpret_cast<uint32_t*>(out + col0 + d * 8) = pack_bf16x2(o[mt][d][2 * h] * f * gate_of(a, t, col0 + d * 8), o[mt][d][2 * h + 1] * f * gate_of(a, t, col0 + d * 8 + 1));
      }
    return;
  }

  // each warp's sums, maxima and denominators to shared memory; then one owner a (row, column) over the warps and the cluster
  float *so = reinterpret_cast<float*>(smem + S::O), *sml = reinterpret_cast<float*>(smem + S::ML);  // [WK][ROWS]
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
  __syncthreads();
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
    __syncthreads();
    float mm = -INFINITY, ll = 0.f;
    if (tid < rows) {
#pragma unroll
      for (int w = 0; w < WK; ++w) mm = fmaxf(mm, sml[(w * ROWS + tid) * 2]);
      const float m = mm == -INFINITY ? 0.f : mm;
#pragma unroll
      for (int w = 0; w < WK; ++w) ll += sml[(w * ROWS + tid) * 2 + 1] * exp2_of(sml[(w * ROWS + tid) * 2] - m);
      sml[tid * 2] = mm, sml[tid * 2 + 1] = ll;
    }
    __syncthreads();
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
    static_cast<uint16_t*>(a.out)[t * a.ld_o + col] = (uint16_t)float_to_bf16_bits(l > 0.f ? acc / l * gate : 0.f);
  }
  if (splits > 1) cluster_barrier();  // the others have read this CTA's part
}

template <int DK, int DV, int WR, int WK, int MT>
static int launch_heads(HeadsArgs a, cudaStream_t s) {
  using S = HeadsShape<DK, DV, WR, WK, MT>;
  a.entries = a.chunk ? 1 : (int)a.T, a.pairs = a.chunk ? (int)a.T * a.rep : a.rep, a.tiles = (int)ceil_div(a.pairs, S::ROWS);
  // the keys over a cluster's CTAs where the tiles alone leave SMs idle: about two CTAs an SM in flight, two tiles of keys a CTA
  const int64_t ctas = (int64_t)a.kv_heads * a.entries * a.tiles;
  int splits = 1;
  while (splits < 8 && ctas * splits * 2 <= 4 * 148 && a.seen >= 4 * HA_KEYS * splits) splits *= 2;
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(heads_attention_kernel<DK, DV, WR, WK, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::SMEM);
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3((unsigned)splits, (unsigned)a.kv_heads, (unsigned)(a.entries * a.tiles)), cfg.blockDim = dim3(32 * WR * WK);
  cfg.dynamicSmemBytes = S::SMEM, cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = (unsigned)splits, attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr, cfg.numAttrs = splits > 1 ? 2 : 1;
  cudaLaunchKernelEx(&cfg, heads_attention_kernel<DK, DV, WR, WK, MT>, a);
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

// ---- any sizes, bf16 or fp32: a CTA per token and eight heads, a warp a head.  A lane owns a key for the scores and every
// 32nd column for the sum; keys and values are read where they are.
constexpr int PLAIN_HEADS = 8, PLAIN_COLS = 32;

template <typename Act, int COLS>
__global__ void __launch_bounds__(32 * PLAIN_HEADS) heads_attention_plain_kernel(const HeadsArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ float plain_q[];  // [8][dim]
  const int64_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y * PLAIN_HEADS + warp, W = a.dim + a.vdim;
  if (h >= a.heads) return;
  const int64_t seq = (a.base ? a.base[t] : 0) + a.row0, room = seq < 0 ? 0 : a.cache_rows - seq;
  const int place = a.last[t], keys = (int)max((int64_t)0, min((int64_t)place + 1, room)), lo = span_start(place, a.span);
  const Act* cache = static_cast<const Act*>(a.cache) + (h / a.rep) * a.head_stride;
  float* q = plain_q + warp * a.dim;
  for (int c = lane; c < a.dim; c += 32) q[c] = value_of(static_cast<const Act*>(a.q)[t * a.ld_q + (int64_t)h * a.dim + c]);
  __syncwarp();
  float acc[COLS];
#pragma unroll
  for (int i = 0; i < COLS; ++i) acc[i] = 0.f;
  float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f;
  for (int k0 = lo; k0 < keys; k0 += 32) {
    const int n = min(32, keys - k0);
    const Act* rows = cache + (seq + k0) * W;
    float s = -INFINITY;
    if (lane < n) {
      s = 0.f;
      for (int c = 0; c < a.dim; ++c) s = fmaf(q[c], value_of(rows[(int64_t)lane * W + c]), s);
      s *= a.scale;
    }
    const float m_new = fmaxf(m, warp_max(s)), corr = expf(m - m_new), p = lane < n ? expf(s - m_new) : 0.f;
    m = m_new, l = l * corr + warp_sum(p);
#pragma unroll
    for (int i = 0; i < COLS; ++i) acc[i] *= corr;
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const Act* v = rows + (int64_t)j * W + a.dim;
#pragma unroll
      for (int i = 0; i < COLS; ++i)
        if (i * 32 + lane < a.vdim) acc[i] = fmaf(pj, value_of(v[i * 32 + lane]), acc[i]);
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
  for (int i = 0; i < COLS; ++i) {
    const int64_t col = (int64_t)h * a.vdim + i * 32 + lane;
    if (i * 32 + lane < a.vdim) store_value(static_cast<Act*>(a.out) + t * a.ld_o + col, acc[i] * inv * gate_of(a, t, col));
  }
}

template <typename Act, int COLS>
static int launch_plain(const HeadsArgs& a, cudaStream_t s) {
  const size_t smem = (size_t)PLAIN_HEADS * a.dim * sizeof(float);
  return launch_after(heads_attention_plain_kernel<Act, COLS>, dim3((unsigned)a.T, (unsigned)ceil_div(a.heads, PLAIN_HEADS)), dim3(32 * PLAIN_HEADS), smem, s, "fb_heads_attention", a);
}

}  // namespace fb

extern "C" int fb_heads_attention(int dtype, const void* q, int64_t T, int64_t ld_q, int heads, int kv_heads, int dim, int vdim, const void* cache, int64_t cache_rows,
                                  int64_t head_stride, const int32_t* base, int64_t row0, const int32_t* last, int64_t max_keys, int chunk, int span, float scale,
                                  const float* sink, int gate_dtype, const void* gate, int64_t ld_g, void* out, int64_t ld_o, void* stream) {
  using namespace fb;
  FB_REQUIRE(q && cache && last && out && T >= 1 && max_keys >= 1 && cache_rows >= 1, "fb_heads_attention: null pointer or empty");
  FB_REQUIRE(heads >= 1 && kv_heads >= 1 && heads % kv_heads == 0 && dim >= 1 && vdim >= 1 && kv_heads <= 65535, "fb_heads_attention: whole groups of query heads per key head (got %d / %d)", heads, kv_heads);
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "fb_heads_attention: bf16 or fp32 rows");
  FB_REQUIRE(dim <= 1024 && vdim <= 32 * PLAIN_COLS, "fb_heads_attention: heads of up to 1024 columns (got %d and %d)", dim, vdim);
  FB_REQUIRE(ld_q >= (int64_t)heads * dim && ld_o >= (int64_t)heads * vdim && head_stride >= cache_rows * (dim + vdim) && row0 >= 0 && span >= 0, "fb_heads_attention: row strides too small");
  FB_REQUIRE(!gate || ((gate_dtype == FB_BF16 || gate_dtype == FB_FP32) && ld_g >= (int64_t)heads * vdim), "fb_heads_attention: gates, bf16 or fp32, one a column of the result");
  FB_REQUIRE(!chunk || !base, "fb_heads_attention: a chunk is one sequence's (no base)");
  HeadsArgs a{q, T, ld_q, heads, kv_heads, dim, vdim, heads / kv_heads, cache, cache_rows, head_stride, base, last, row0, chunk, span, scale, sink, gate_dtype, gate, ld_g, out, ld_o, span > 0 && span < max_keys ? span : max_keys, 0, 0, 0};
  const auto s = (cudaStream_t)stream;
  const bool pieces = dim % 8 == 0 && vdim % 8 == 0 && ld_q % 8 == 0 && head_stride % 8 == 0 && ld_o % 2 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)cache % 16 == 0 && (uintptr_t)out % 4 == 0;
  if (dtype == FB_FP32) return vdim <= 256 ? launch_plain<float, 8>(a, s) : launch_plain<float, PLAIN_COLS>(a, s);
  if (pieces && scale > 0.f && heads_prompt_supports(a)) return heads_prompt(a, s);
  const int64_t most = chunk ? ceil_div(T * a.rep, 64) : T * ceil_div(a.rep, 16);  // (of tiles: a grid's limit)
  if (!pieces || !(scale > 0.f) || dim > 256 || vdim > 256 || most > 65535) return vdim <= 256 ? launch_plain<uint16_t, 8>(a, s) : launch_plain<uint16_t, PLAIN_COLS>(a, s);
  return dim <= 64 ? launch_values<64>(a, s) : dim <= 96 ? launch_values<96>(a, s) : dim <= 128 ? launch_values<128>(a, s) : dim <= 192 ? launch_values<192>(a, s) : launch_values<256>(a, s);
}
