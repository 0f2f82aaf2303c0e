// Attention over a cache of latents: a cache row is a token's normed latent (kv_rank columns) and one rotated key part
// (rot columns) that all heads share.  A head's query is taken into the latent's space before (q W_uk), so its score is one
// dot product with the whole row and its output the weighted sum of the rows' latents; the values' matrix follows after.
// Every head reads the same row, so a row is read once for all of them.
//
//   fb_latent_put        what follows the joint down-projection: RMSNorm of the query latent (or, of a design without one, the
//                        queries taken apart and turned) and of the key-value latent, rotation of the shared key part, the new
//                        row into the cache
//   fb_rotate_pairs      neighbouring columns (2i, 2i + 1) of each head turned by the token's angle
//   fb_latent_attention  softmax, within a window if there is one, with an optional sink per head (one more term of the denominator); bf16 rows of suitable
//                        sizes on the tensor cores (latent_tcgen05.cu), everything else - fp32, odd sizes - here
#include "latent.cuh"
#include "launch.cuh"
#include "values.cuh"

namespace fb {

struct LatentPutArgs {
  const void* down;  // [T, ld]: query latent (q_rank, may be 0), key-value latent (kv_rank), key part (rot)
  int64_t ld;
  int q_rank, kv_rank, rot, dims;  // the first `dims` of the key part turn
  const float *q_norm, *kv_norm;
  float eps;
  const double* freq;  // [dims / 2]
  float mag;
  const int32_t *places, *rows;
  void* q_out;  // [T, ld_q]
  int64_t ld_q;
  int heads, dim;  // heads > 0: the row begins with heads x (dim | rot) instead of a query latent
  void* q_turned;  // head h of token t at t * ld_turned + h * turned_head
  int64_t ld_turned, turned_head;
  int per, fours;  // heads a block; all of that in whole, aligned groups of four columns
  void* cache;  // [cache_rows, kv_rank + rot]
  int64_t cache_rows;
};

template <typename In, typename Act>
__global__ void __launch_bounds__(256) latent_put_kernel(const LatentPutArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const In* x = static_cast<const In*>(a.down) + t * a.ld;
  extern __shared__ float put_turns[];  // [dims / 2] cos, [dims / 2] sin
  const int half = a.dims / 2;
  if (a.heads && blockIdx.y + 1 < gridDim.y) {  // queries: the plain parts side by side, the others turned
    const int h0 = blockIdx.y * a.per, h1 = min(a.heads, h0 + a.per), W = a.dim + a.rot, pairs = (a.rot + 1) / 2, place = a.places[t];
    Act* plain = static_cast<Act*>(a.q_out) + t * a.ld_q;
    if (a.fours) {  // (a thread makes the turn of its own columns)
      const int groups = W / 4;
      for (int j = threadIdx.x; j < (h1 - h0) * groups; j += blockDim.x) {
        const int h = h0 + j / groups, c = 4 * (j % groups);
        float4 v = four(x + h * W + c);
        if (c < a.dim) {
          put_four(plain + h * a.dim + c, v);
          continue;
        }
        const int r = c - a.dim;
        float cs, sn;
        if (r < a.dims) {
          turn_of(place, a.freq[r / 2], a.mag, cs, sn);
          v = make_float4(v.x * cs - v.y * sn, v.y * cs + v.x * sn, v.z, v.w);
        }
        if (r + 2 < a.dims) {
          turn_of(place, a.freq[r / 2 + 1], a.mag, cs, sn);
          v = make_float4(v.x, v.y, v.z * cs - v.w * sn, v.w * cs + v.z * sn);
        }
        put_four(static_cast<Act*>(a.q_turned) + t * a.ld_turned + h * a.turned_head + r, v);
      }
      return;
    }
    for (int i = threadIdx.x; i < half; i += blockDim.x) turn_of(place, a.freq[i], a.mag, put_turns[i], put_turns[half + i]);
    __syncthreads();
    for (int i = h0 * a.dim + threadIdx.x; i < h1 * a.dim; i += blockDim.x) store_value(plain + i, value_of(x[i / a.dim * W + i % a.dim]));
    for (int j = threadIdx.x; j < (h1 - h0) * pairs; j += blockDim.x) {
      const int h = h0 + j / pairs, i = j % pairs;
      const bool two = 2 * i + 1 < a.rot;
      const In* from = x + h * W + a.dim + 2 * i;
      Act* out = static_cast<Act*>(a.q_turned) + t * a.ld_turned + h * a.turned_head + 2 * i;
      const float u = value_of(from[0]), v = two ? value_of(from[1]) : 0.f;
      store_value(out, i < half ? u * put_turns[i] - v * put_turns[half + i] : u);
      if (two) store_value(out + 1, i < half ? v * put_turns[i] + u * put_turns[half + i] : v);
    }
    return;
  }
  if (blockIdx.y == 0 && !a.heads) {  // the query latent
    float ss = 0.f;
    for (int c = threadIdx.x; c < a.q_rank; c += blockDim.x) ss = fmaf(value_of(x[c]), value_of(x[c]), ss);
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)a.q_rank + a.eps);
    Act* out = static_cast<Act*>(a.q_out) + t * a.ld_q;
    for (int c = threadIdx.x; c < a.q_rank; c += blockDim.x) store_value(out + c, value_of(x[c]) * r * a.q_norm[c]);
    return;
  }
  const int64_t row = a.rows[t];
  if (row < 0 || row >= a.cache_rows) return;  // (the whole block: nothing is written outside the cache)
  x += a.heads ? a.heads * (a.dim + a.rot) : a.q_rank;
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.kv_rank; c += blockDim.x) ss = fmaf(value_of(x[c]), value_of(x[c]), ss);
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)a.kv_rank + a.eps);
  Act* out = static_cast<Act*>(a.cache) + row * (a.kv_rank + a.rot);
  for (int c = threadIdx.x; c < a.kv_rank; c += blockDim.x) store_value(out + c, value_of(x[c]) * r * a.kv_norm[c]);
  x += a.kv_rank, out += a.kv_rank;
  const int place = a.places[t];
  for (int i = threadIdx.x; i < a.dims / 2; i += blockDim.x) {
    float c, s;
    turn_of(place, a.freq[i], a.mag, c, s);
    const float u = value_of(x[2 * i]), v = value_of(x[2 * i + 1]);
    store_value(out + 2 * i, u * c - v * s), store_value(out + 2 * i + 1, v * c + u * s);
  }
  for (int c = a.dims + threadIdx.x; c < a.rot; c += blockDim.x) store_value(out + c, value_of(x[c]));
}

struct RotateArgs {
  const void* x;  // head h of token t at x + t * x_row + h * x_head
  int64_t x_row, x_head;
  void* out;
  int64_t o_row, o_head;
  int heads, width, dims;
  const double* freq;
  float mag;
  const int32_t* places;
};

// a block per token; the angles are made once and kept in shared memory for all the heads
template <typename Act>
__global__ void __launch_bounds__(512) rotate_pairs_kernel(const RotateArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ float turns[];  // [dims / 2] cos, [dims / 2] sin
  const int64_t t = blockIdx.x;
  const int half = a.dims / 2, place = a.places[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) turn_of(place, a.freq[i], a.mag, turns[i], turns[half + i]);
  __syncthreads();
  const int pairs = (a.width + 1) / 2;
  for (int j = threadIdx.x; j < a.heads * pairs; j += blockDim.x) {
    const int h = j / pairs, i = j % pairs;
    const Act* x = static_cast<const Act*>(a.x) + t * a.x_row + h * a.x_head + 2 * i;
    Act* out = static_cast<Act*>(a.out) + t * a.o_row + h * a.o_head + 2 * i;
    const float u = value_of(x[0]), v = 2 * i + 1 < a.width ? value_of(x[1]) : 0.f;
    if (i < half) {
      store_value(out, u * turns[i] - v * turns[half + i]), store_value(out + 1, v * turns[i] + u * turns[half + i]);
    } else {
      store_value(out, u);
      if (2 * i + 1 < a.width) store_value(out + 1, v);
    }
  }
}

// ---- attention, any sizes, bf16 or fp32: a CTA per token and eight heads, a warp a head.  Tiles of 32 cache rows are
// widened into shared memory; a lane owns a key for the scores and every 32nd latent column for the sum.
constexpr int LAT_HEADS = 8, LAT_KEYS = 32, LAT_COLS = 32;  // (LAT_COLS * 32 = 1024: the widest latent)

template <typename Act, int COLS>
__global__ void __launch_bounds__(32 * LAT_HEADS) latent_attention_kernel(const LatentArgs a) {
  griddep_launch_dependents();
  griddep_wait();
  extern __shared__ float lat_smem[];
  const int W = a.rank + a.rot, pitch = W | 1;
  float* sk = lat_smem;                    // [32][pitch]
  float* sq = sk + LAT_KEYS * pitch;       // [8][W]
  const int64_t t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y * LAT_HEADS + warp;
  const bool on = h < a.heads;
  const Act* cache = static_cast<const Act*>(a.cache);
  const int64_t first = (a.base ? a.base[t] : 0) + a.row0;
  const int64_t room = first < 0 ? 0 : a.cache_rows - first;
  const int keys = (int)max((int64_t)0, min((int64_t)a.last[t] + 1, room)), lo = a.window > 0 ? max(0, a.last[t] - a.window + 1) : 0;
  if (on) {
    const Act* q = static_cast<const Act*>(a.q) + t * a.ld_q + (int64_t)h * W;
    for (int c = lane; c < W; c += 32) sq[warp * W + c] = value_of(q[c]);
  }
  float acc[COLS];
#pragma unroll
  for (int i = 0; i < COLS; ++i) acc[i] = 0.f;
  float m = a.sink && on ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f;  // the sink: a key of its own with no value
  for (int k0 = lo; k0 < keys; k0 += LAT_KEYS) {
    const int n = min(LAT_KEYS, keys - k0);
    __syncthreads();
    for (int i = threadIdx.x; i < n * W; i += blockDim.x) sk[(i / W) * pitch + i % W] = value_of(cache[(first + k0 + i / W) * W + i % W]);
    __syncthreads();
    if (!on) continue;
    float s = -INFINITY;
    if (lane < n) {
      s = 0.f;
      const float *kr = sk + lane * pitch, *qr = sq + warp * W;
      for (int c = 0; c < W; ++c) s = fmaf(qr[c], kr[c], s);
      s *= a.scale;
    }
    const float m_new = fmaxf(m, warp_max(s)), corr = expf(m - m_new), p = lane < n ? expf(s - m_new) : 0.f;
    m = m_new, l = l * corr + warp_sum(p);
#pragma unroll
    for (int i = 0; i < COLS; ++i) acc[i] *= corr;
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const float* kr = sk + j * pitch;
#pragma unroll
      for (int i = 0; i < COLS; ++i)
        if (i * 32 + lane < a.rank) acc[i] = fmaf(pj, kr[i * 32 + lane], acc[i]);
    }
  }
  if (!on) return;
  Act* out = static_cast<Act*>(a.out) + t * a.ld_o + (int64_t)h * a.rank;
  const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
  for (int i = 0; i < COLS; ++i)
    if (i * 32 + lane < a.rank) store_value(out + i * 32 + lane, acc[i] * inv);
}

template <typename Act, int COLS>
static int launch_latent(const LatentArgs& a, cudaStream_t s) {
  const int W = a.rank + a.rot;
  const size_t smem = (size_t)(LAT_KEYS * (W | 1) + LAT_HEADS * W) * sizeof(float);
  FB_REQUIRE(smem <= 220 * 1024, "fb_latent_attention: rows of %d columns are too wide", W);
  static std::atomic<uint64_t> opted{0};
  if (first_on_device(opted)) cudaFuncSetAttribute(latent_attention_kernel<Act, COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  latent_attention_kernel<Act, COLS><<<dim3((unsigned)a.T, (unsigned)ceil_div(a.heads, LAT_HEADS)), 32 * LAT_HEADS, smem, s>>>(a);
  return launch_status("fb_latent_attention");
}

}  // namespace fb

extern "C" int fb_latent_put(int in_dtype, const void* down, int64_t T, int64_t ld, int q_rank, int kv_rank, int rot, int dims, const float* q_norm,
                             const float* kv_norm, float eps, const double* freq, float mag, const int32_t* places, const int32_t* rows, int dtype,
                             void* q_out, int64_t ld_q, int heads, int dim, void* q_turned, int64_t ld_turned, int64_t turned_head, void* cache, int64_t cache_rows, void* stream) {
  FB_REQUIRE(down && kv_norm && freq && places && rows && cache && T >= 1 && kv_rank >= 1, "fb_latent_put: null pointer or empty");
  FB_REQUIRE(q_rank >= 0 && (q_rank == 0 || (q_norm && q_out && ld_q >= q_rank)), "fb_latent_put: a query latent takes its norm and somewhere to go");
  FB_REQUIRE(heads >= 0 && (heads == 0 || (q_rank == 0 && dim >= 1 && q_out && ld_q >= (int64_t)heads * dim && (rot == 0 || q_turned))), "fb_latent_put: queries take somewhere for both their parts, and no query latent");
  FB_REQUIRE(rot >= 0 && dims >= 0 && dims % 2 == 0 && dims <= rot && dims <= 8192 && ld >= q_rank + (int64_t)heads * (dim + rot) + kv_rank + rot && cache_rows >= 1, "fb_latent_put: the turned columns are an even number within the key part");
  FB_REQUIRE((in_dtype == FB_BF16 || in_dtype == FB_FP32) && (dtype == FB_BF16 || dtype == FB_FP32), "fb_latent_put: bf16 or fp32");
  fb::LatentPutArgs a{down, ld, q_rank, kv_rank, rot, dims, q_norm, kv_norm, eps, freq, mag, places, rows, q_out, ld_q, heads, dim, q_turned, ld_turned, turned_head, 0, 0, cache, cache_rows};
  const auto s = (cudaStream_t)stream;
  FB_REQUIRE(in_dtype == FB_FP32 || dtype == FB_BF16, "fb_latent_put: fp32 results come from fp32");
  auto whole = [](const void* p, int64_t ld, int64_t step, int bytes) { return (uintptr_t)p % (4 * bytes) == 0 && ld % 4 == 0 && step % 4 == 0; };
  const int in_bytes = in_dtype == FB_FP32 ? 4 : 2, bytes = dtype == FB_FP32 ? 4 : 2;
  a.per = heads && 1024 / (dim + rot) > 1 ? 1024 / (dim + rot) : 1;
  a.fours = dim % 4 == 0 && rot % 4 == 0 && whole(down, ld, 0, in_bytes) && whole(q_out, ld_q, 0, bytes) && whole(q_turned, ld_turned, turned_head, bytes);
  const dim3 grid((unsigned)T, 1u + (heads ? (unsigned)fb::ceil_div(heads, a.per) : 1u)), block(256);
  const size_t smem = heads ? dims * sizeof(float) : 0;
  if (in_dtype == FB_FP32 && dtype == FB_FP32) return fb::launch_after(fb::latent_put_kernel<float, float>, grid, block, smem, s, "fb_latent_put", a);
  if (in_dtype == FB_FP32) return fb::launch_after(fb::latent_put_kernel<float, uint16_t>, grid, block, smem, s, "fb_latent_put", a);
  return fb::launch_after(fb::latent_put_kernel<uint16_t, uint16_t>, grid, block, smem, s, "fb_latent_put", a);
}

extern "C" int fb_rotate_pairs(int dtype, const void* x, int64_t T, int heads, int64_t x_row, int64_t x_head, int width, int dims, const double* freq,
                               float mag, const int32_t* places, void* out, int64_t o_row, int64_t o_head, void* stream) {
  FB_REQUIRE(x && out && freq && places && T >= 1 && heads >= 1 && width >= 1, "fb_rotate_pairs: null pointer or empty");
  FB_REQUIRE(dims >= 0 && dims % 2 == 0 && dims <= width && dims <= 8192, "fb_rotate_pairs: an even number of a head's columns turn");
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "fb_rotate_pairs: bf16 or fp32");
  fb::RotateArgs a{x, x_row, x_head, out, o_row, o_head, heads, width, dims, freq, mag, places};
  if (dtype == FB_FP32) fb::rotate_pairs_kernel<float><<<(unsigned)T, 512, dims * 4, (cudaStream_t)stream>>>(a);
  else fb::rotate_pairs_kernel<uint16_t><<<(unsigned)T, 512, dims * 4, (cudaStream_t)stream>>>(a);
  return fb::launch_status("fb_rotate_pairs");
}

extern "C" size_t fb_latent_attention_workspace_bytes(int dtype, int64_t T, int heads, int rank, int rot, int64_t max_keys, int chunk, int window) {
  return dtype == FB_BF16 && heads >= 1 && rank >= 1 && rot >= 0 ? fb::latent_tcgen05_workspace(T, heads, rank, rot, max_keys, chunk, window) : 0;
}

extern "C" int fb_latent_attention(int dtype, const void* q, int64_t T, int64_t ld_q, int heads, int rank, int rot, const void* cache, int64_t cache_rows,
                                   const int32_t* base, int64_t row0, const int32_t* last, int64_t max_keys, int chunk, int window, float scale, const float* sink,
                                   void* out, int64_t ld_o, void* workspace, size_t workspace_bytes, void* stream) {
  FB_REQUIRE(q && cache && last && out && T >= 1 && heads >= 1 && rank >= 1 && rot >= 0 && max_keys >= 1, "fb_latent_attention: null pointer or empty");
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "fb_latent_attention: bf16 or fp32 rows");
  FB_REQUIRE(ld_q >= (int64_t)heads * (rank + rot) && ld_o >= (int64_t)heads * rank && cache_rows >= 1 && row0 >= 0 && window >= 0, "fb_latent_attention: row strides too small");
  FB_REQUIRE(rank <= 32 * fb::LAT_COLS, "fb_latent_attention: latents of up to %d columns", 32 * fb::LAT_COLS);
  fb::LatentArgs a{q, T, ld_q, heads, rank, rot, cache, cache_rows, base, row0, last, max_keys, window, chunk, scale, sink, out, ld_o, workspace, workspace_bytes};
  const auto s = (cudaStream_t)stream;
  if (dtype == FB_BF16 && fb::latent_tcgen05_supports(a)) return fb::latent_tcgen05(a, s);
  if (dtype == FB_FP32) return rank <= 256 ? fb::launch_latent<float, 8>(a, s) : fb::launch_latent<float, fb::LAT_COLS>(a, s);
  return rank <= 256 ? fb::launch_latent<uint16_t, 8>(a, s) : fb::launch_latent<uint16_t, fb::LAT_COLS>(a, s);
}
