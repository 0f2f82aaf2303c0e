// Attention with grouped key heads over a cache whose rows are a key and then its value: the two may differ in width, the
// keys a token sees may be confined to its own span of the sequence (spans of `span` places, counted from its start) or to the
// last `window` places, scores may be capped, a number per head may join the softmax's denominator, and the output may be gated
// column by column.  Or there is no softmax: a key's weight is a sigmoid of its own score and a number of the head.
//
// A CTA has one key head, a tile of (token, query head) pairs that share it - the pairs of one token in a decode step, those
// of consecutive tokens in a prompt's chunk - and a run of the keys that they see; tiles of 64 keys and their values come in by
// TMA, asked for by a warp of its own, a ring of up to six; q k^T and p v run on mma.sync with an online softmax in registers.
//   prompt   128 pairs (values of more than 128 columns: 64), a warp 32 of them over all keys of a tile
//   decode   16 pairs, a warp a quarter of a tile's keys; merged in shared memory
// The runs of one tile's keys are a cluster's CTAs: their parts are merged over distributed shared memory, so no result
// passes through global memory and there is no second kernel.  A prompt with tiles enough goes to heads_prompt.cu.
//
// bf16 rows of whole 16-byte pieces, heads of up to 256 columns; everything else (fp32, odd or wider heads) takes a plain
// kernel at the end of the file.  Every wait is bounded (sm100.cuh).
#include "heads.cuh"
#include "launch.cuh"
#include "tma_host.cuh"

namespace fb {

// heads_attention_64.cu ...: keys of up to so many columns
int heads_attention_64(const HeadsArgs& a, cudaStream_t s);
int heads_attention_128(const HeadsArgs& a, cudaStream_t s);
int heads_attention_192(const HeadsArgs& a, cudaStream_t s);
int heads_attention_256(const HeadsArgs& a, cudaStream_t s);

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
  const int place = a.last[t], keys = (int)max((int64_t)0, min((int64_t)place + 1, room)), lo = first_seen(a, place);
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
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    }
    if (a.key_bias) {
      m = 0.f, l = 1.f;
      s = lane < n ? sigmoid_f(s + a.key_bias[h]) : 0.f;
    }
    float corr = 1.f, p = s;
    if (!a.key_bias) {
      const float m_new = fmaxf(m, warp_max(s));
      corr = expf(m - m_new), p = lane < n ? expf(s - m_new) : 0.f;
      m = m_new, l = l * corr + warp_sum(p);
    }
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
  const float inv = l > 0.f ? a.out_scale / l : 0.f;
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
                                  int64_t head_stride, const int32_t* base, int64_t row0, const int32_t* last, int64_t max_keys, int chunk, int span, int window, float scale,
                                  float softcap, const float* sink, const float* key_bias, float out_scale, int gate_dtype, const void* gate, int64_t ld_g, void* out, int64_t ld_o, void* stream) {
  using namespace fb;
  FB_REQUIRE(q && cache && last && out && T >= 1 && max_keys >= 1 && cache_rows >= 1, "fb_heads_attention: null pointer or empty");
  FB_REQUIRE(heads >= 1 && kv_heads >= 1 && heads % kv_heads == 0 && dim >= 1 && vdim >= 1 && kv_heads <= 65535, "fb_heads_attention: whole groups of query heads per key head (got %d / %d)", heads, kv_heads);
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "fb_heads_attention: bf16 or fp32 rows");
  FB_REQUIRE(dim <= 1024 && vdim <= 32 * PLAIN_COLS, "fb_heads_attention: heads of up to 1024 columns (got %d and %d)", dim, vdim);
  FB_REQUIRE(ld_q >= (int64_t)heads * dim && ld_o >= (int64_t)heads * vdim && head_stride >= cache_rows * (dim + vdim) && row0 >= 0 && span >= 0 && window >= 0, "fb_heads_attention: row strides too small");
  FB_REQUIRE(!gate || ((gate_dtype == FB_BF16 || gate_dtype == FB_FP32) && ld_g >= (int64_t)heads * vdim), "fb_heads_attention: gates, bf16 or fp32, one a column of the result");
  FB_REQUIRE(!chunk || !base, "fb_heads_attention: a chunk is one sequence's (no base)");
  FB_REQUIRE(softcap >= 0.f, "fb_heads_attention: a cap of scores is positive (0: none)");
  FB_REQUIRE(!key_bias || !sink, "fb_heads_attention: a sink joins a softmax's denominator");
  HeadsArgs a{q, T, ld_q, heads, kv_heads, dim, vdim, heads / kv_heads, cache, cache_rows, head_stride, base, last, row0, chunk, span, window, scale, softcap, sink, key_bias, out_scale, gate_dtype, gate, ld_g, out, ld_o, max_keys, 0, 0, 0, 0};
  if (span > 0 && span < a.seen) a.seen = span;
  if (window > 0 && window + (chunk ? ceil_div(128, a.rep) : 0) < a.seen) a.seen = window + (chunk ? ceil_div(128, a.rep) : 0);  // (a tile's tokens' windows together)
  const auto s = (cudaStream_t)stream;
  const bool pieces = dim % 8 == 0 && vdim % 8 == 0 && ld_q % 8 == 0 && head_stride % 8 == 0 && ld_o % 2 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)cache % 16 == 0 && (uintptr_t)out % 4 == 0;
  if (dtype == FB_FP32) return vdim <= 256 ? launch_plain<float, 8>(a, s) : launch_plain<float, PLAIN_COLS>(a, s);
  if (pieces && scale > 0.f && heads_prompt_supports(a)) return heads_prompt(a, s);
  const int64_t most = chunk ? ceil_div(T * a.rep, 64) : T * ceil_div(a.rep, 16);  // (of tiles: a grid's limit)
  if (!pieces || !(scale > 0.f) || dim > 256 || vdim > 256 || most > 65535 || cache_rows >= (1ll << 31) || tma_encoder() == nullptr) return vdim <= 256 ? launch_plain<uint16_t, 8>(a, s) : launch_plain<uint16_t, PLAIN_COLS>(a, s);
  return dim <= 64 ? heads_attention_64(a, s) : dim <= 128 ? heads_attention_128(a, s) : dim <= 192 ? heads_attention_192(a, s) : heads_attention_256(a, s);
}
