/* ferrite_b200: C ABI of the B200 (sm_100a) decode hot path.
 *
 * This is the boundary a host binds instead of ferrite's Tensix code generator: every
 * entry point replaces one device kernel ferrite's `Tensor` launches through
 * `Runtime.launch` (ferrite/runtime.py:373-378).  The reference's own FFI is ctypes to a
 * shared library with plain integer/pointer arguments (ferrite/pci.py:19-31); this header
 * keeps that style: device pointers, sizes, a CUDA stream, an int status.
 *
 * Conventions
 *   - every pointer is a DEVICE pointer unless its name ends in `_host`;
 *   - `stream` is a cudaStream_t passed as void*; launches are asynchronous on it and
 *     nothing here synchronises, so a sequence of calls can be captured in a CUDA graph
 *     (the analogue of ferrite's `jit` replay, ferrite/tensor.py:788-810);
 *   - a function returns FB_OK (0) or a negative fb_status; fb_last_error() gives the
 *     reason as text (calling thread's last failure);
 *   - matrices are row-major; `bf16` means the 16-bit pattern ferrite uploads
 *     (round to nearest even, ferrite/tensor.py:56).
 *
 * Packed block-float matrix [K, N] (N a multiple of 16), format FB_BFP8 or FB_BFP4.
 * The values are exactly those of ferrite's block floats (models/gpt2.py:21-32,
 * ferrite/compiler.py:15-20,1631-1684): each run of 16 consecutive columns of one row k
 * shares the largest biased bf16 exponent of the run (`top`), every value keeps a sign and
 * a 7-bit (bfp8) or 3-bit (bfp4) magnitude, value = +-mag * 2^(top-133) (bfp4: mag*16).
 * The footprint is ferrite's too: 1088 / 576 bytes per 1024 values.  The byte ORDER is
 * this library's own (ferrite's is its 32x32 Tensix tile with 16x16 faces): a matrix is a
 * grid of UNITS of 64 rows of K x 64 columns (4 runs); rows and columns are padded with
 * zeros up to whole units (ferrite pads its tiles the same way, ferrite/tensor.py:22-24).
 *     unit (g, s) for column group g = n/64 and row step s = k/64 lies at byte
 *       (g * ceil(K/64) + s) * U,   U = 4352 (bfp8) or 2304 (bfp4);
 *     the units of one column group follow each other along K, so a stretch of K of one
 *     group is one contiguous piece of memory;
 *     inside a unit, for run r = (n/16)%4 and row i = k%64:
 *       mantissas  bfp8: 16 bytes at (r*64 + i)*16, four little-endian 32-bit words of four columns each;
 *                         in word h (columns c0..c3 = 4h..4h+3 of the run):
 *                           byte0 = mag(c0) | sign(c3)<<7   byte1 = mag(c2) | sign(c0)<<7
 *                           byte2 = mag(c1) | sign(c2)<<7   byte3 = mag(c3) | sign(c1)<<7
 *                  bfp4:  8 bytes at (r*64 + i)*8, two words of eight columns each; nibble p (bits 4p..4p+3)
 *                         = mag3(v_p) | sign(v_((p+5) mod 8))<<3 with v_p = column 2*(p%4) + p/4 of the word.
 *                  (A value's sign is parked one byte / three nibbles above its magnitude, cyclically, so a mask of
 *                  the word, or of the word rotated, is two bf16 subnormals mag * 2^-133 with their signs in place;
 *                  two exact multiplications by powers of two then give +-mag * 2^(top-133).)
 *       exponents  one byte at 4*64*(16|8) + r*64 + i.
 *   A zero magnitude is stored without a sign (as ferrite stores it).  fb_unpack_fields
 *   returns (top, sign, mag) per value for checking against the reference model.
 *   A batch of matrices (a mixture's experts) is that many packed matrices back to back,
 *   fb_packed_bytes(fmt, K, N) apart.
 */
#ifndef FERRITE_B200_H
#define FERRITE_B200_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef enum {
  FB_OK = 0,
  FB_ERR_ARG = -1,     /* shape / dtype / alignment misuse: what ferrite asserts on (e.g. tensor.py:122,133-136) */
  FB_ERR_LAUNCH = -2,  /* a CUDA launch or runtime call failed */
  FB_ERR_TIMEOUT = -3, /* a bounded device wait gave up (ferrite: TimeoutError, runtime.py:466-484) */
  FB_ERR_MEMORY = -4   /* a caller-provided workspace is too small (ferrite: MemoryError, runtime.py:445) */
} fb_status;

/* dtype names follow ferrite's Tensor.dtype strings (ferrite/tensor.py:17) */
typedef enum { FB_BF16 = 0, FB_FP32 = 1, FB_INT32 = 2, FB_BFP8 = 3, FB_BFP4 = 4 } fb_dtype;

/* what a matmul fuses after its accumulation */
typedef enum {
  FB_EPI_NONE = 0,
  FB_EPI_SWIGLU = 1,   /* out[t, j] = silu(acc[t, j]) * acc[t, j + N/2]  (models/llama.py:266-275) */
  FB_EPI_RESIDUAL = 2  /* out[t, n] = residual[t, n] + acc[t, n]        (models/llama.py:107-109) */
} fb_epilogue;

int fb_version(void);
const char* fb_last_error(void);
/* Device-side waits are bounded (ferrite gives every wait a timeout, ferrite/chip.py:78-82): a wait that gives up
 * records a non-zero code here and the kernel returns.  Reads and clears it; synchronises with the device. */
int fb_status_word(void);

/* ---- block-float pack / unpack: Tensor.cast("bfp8"|"bfp4") (ferrite/tensor.py:315-320), the packer's
 * bfp8 cast (ferrite/compiler.py:52-70) and bfp4_kernel (ferrite/compiler.py:2038-2072); bit-exact with
 * the numpy model models/gpt2.py:21-32. */
size_t fb_packed_bytes(int fmt, int64_t K, int64_t N);
int fb_quantize(int fmt, const void* src_bf16, int64_t batch, int64_t K, int64_t N, void* dst_packed, void* stream);
/* packed -> bf16 values: what Tensor.tobytes gives for a block float (ferrite/tensor.py:82-107, 718-727) */
int fb_dequantize(int fmt, const void* packed, int64_t batch, int64_t K, int64_t N, void* dst_bf16, void* stream);
/* packed -> top[batch,K,N/16], sign[batch,K,N], mag[batch,K,N] (uint8 each) */
int fb_unpack_fields(int fmt, const void* packed, int64_t batch, int64_t K, int64_t N, uint8_t* top, uint8_t* sign,
                     uint8_t* mag, void* stream);

/* ---- weight matmul: Tensor.matmul with a block-float (or bf16) B (ferrite/tensor.py:443-485,
 * ferrite/compiler.py:699-738), with what models/llama.py computes around it fused in:
 *   x[M, K] bf16 (row stride ldx elements)
 *   optional RMSNorm prologue: h = x * rsqrt(mean(x^2) + eps) * norm_w[K]   (models/llama.py:82-85)
 *   acc = h @ W, fp32 accumulation, W packed [K, N] in `fmt` (FB_BFP8, FB_BFP4 or FB_BF16 row-major)
 *   epilogue (fb_epilogue), out dtype FB_BF16 or FB_FP32 (fp32: the output layer, models/llama.py:479)
 * out is [M, N] (or [M, N/2] after FB_EPI_SWIGLU), row stride ldo elements.
 * M == 1 runs as a bandwidth-bound GEMV on CUDA cores (a CTA per 16 output columns); 2..8 rows of the smaller
 * matrices on tensor-core MMAs whose weight fragments are unpacked in registers; the rest on tcgen05 tensor cores
 * (weight tiles through shared memory, accumulators in TMEM): a CTA per tile of 128 columns (clusters splitting K
 * where the tiles are few), or - with at least a tile per SM and the workspace given - one persistent CTA per SM,
 * the tiles' steps of K shared out evenly (FB_LINEAR_PERSISTENT below).
 * workspace: fb_linear_workspace_bytes(M, K, N) bytes of device scratch (0 / NULL when that is 0):
 * it holds the normalised activations of the RMSNorm prologue between the two kernels of a call, the partial sums of
 * output tiles that several CTAs share, and their arrival counters in the first 18 KB, which every call leaves zero:
 * fb_linear zeroes them itself (in stream order) the first time this process hands it a buffer; nobody else may write
 * there, and a buffer that comes back after other use has to be zeroed by the caller. */
size_t fb_linear_workspace_bytes(int64_t M, int64_t K, int64_t N);
int fb_linear(int fmt, const void* x, int64_t M, int64_t K, int64_t ldx, const void* W, int64_t N, void* out,
              int out_dtype, int64_t ldo, const void* norm_w, float eps, int epilogue, const void* residual,
              int64_t ldr, void* workspace, size_t workspace_bytes, void* stream);

/* Which kernel fb_linear runs (process-wide; for measurements that compare them - results agree within the rounding
 * stated for each).  FB_LINEAR_AUTO (the default) chooses by M as described above; FB_LINEAR_TCGEN05 and
 * FB_LINEAR_GEMV restore the choice without the register-fed kernel (GEMV up to 4 rows when asked for, else one row);
 * FB_LINEAR_MMA sends every shape the register-fed kernel supports (M <= 32, K a multiple of 16) to it, one row too.
 * FB_LINEAR_PERSISTENT runs the tcgen05 path as one persistent CTA per SM, the tiles' steps of K shared out evenly and
 * tiles that several CTAs share summed through the workspace in a fixed order (one row too).
 * FB_LINEAR_GEMV_STREAM runs one row through the streaming GEMV (persistent CTAs fed by bulk copies, each taking an equal
 * stretch of the packed matrix; the output tiles' parts meet in the workspace and are added in a fixed order) or fails
 * with FB_ERR_ARG where its rules do not hold: N a multiple of 64 (128 with SwiGLU), K up to ~13k (the token sits in shared
 * memory as fp32 beside the ring), the workspace given.  Measured slower than the plain GEMV, hence never chosen.
 * The reference has one matmul kernel and no such switch (ferrite/compiler.py:699-738). */
enum fb_linear_kernel { FB_LINEAR_AUTO = 0, FB_LINEAR_TCGEN05 = 1, FB_LINEAR_GEMV = 2, FB_LINEAR_MMA = 3, FB_LINEAR_PERSISTENT = 4, FB_LINEAR_GEMV_STREAM = 5 };
int fb_linear_prefer(int kernel);

/* fb_linear with an RMSNorm handed from the matmul that makes its input to the matmul that consumes it, so that no
 * kernel stands between the two (a decoder block's x + o_proj(...) -> rms -> gate_up, and down_proj -> next block's rms ->
 * qkv: models/llama.py:95-109, 82-85).  No counterpart in the reference, whose fused kernels are generated per tree.
 *   As producer (next_norm_w given; FB_EPI_RESIDUAL or none, out bf16): besides out, xn_out[t, n] = bf16(out[t, n] *
 *   next_norm_w[n]) (rows ld_xn apart) and sumsq_out[part * M + t] = sum over the part's columns of out[t, n]^2, one part
 *   per CTA of the launch: fb_linear_chain_parts(fmt, M, K, N, epilogue) parts (0: this shape cannot chain).
 *   As consumer (sumsq_in given): x is such an xn_out, and the accumulators are scaled by rsqrt(sum of the sumsq_in parts
 *   / K + eps) - what the RMSNorm prologue of fb_linear computes, without its pass over x.
 * A call may be both.  2 <= M <= 128; runs the tcgen05 kernel (a CTA per tile) whatever fb_linear_prefer says. */
int fb_linear_chain_parts(int fmt, int64_t M, int64_t K, int64_t N, int epilogue);
int fb_linear_chained(int fmt, const void* x, int64_t M, int64_t K, int64_t ldx, const void* W, int64_t N, void* out, int out_dtype,
                      int64_t ldo, float eps, int epilogue, const void* residual, int64_t ldr, const float* sumsq_in, int sumsq_parts,
                      const void* next_norm_w, void* xn_out, int64_t ld_xn, float* sumsq_out, void* workspace, size_t workspace_bytes,
                      void* stream);

/* ---- matmul by bf16 weights whose output columns each lie together (W [N, K], as checkpoints store a linear layer): x [M, K]
 * bf16 @ W^T on the tcgen05 tensor cores, fp32 accumulation, with one of these after it: */
enum fb_dense_epilogue_kind {
  FB_DENSE_NONE = 0,
  FB_DENSE_SILU = 1,    /* the first act_cols columns through SiLU */
  FB_DENSE_GLU = 2,     /* W holds gate rows, then as many up rows: out = g sigmoid(slope g) (u + 1), g = min(gate, limit), u = up in -limit .. limit;
                           out is [M, N / 2] */
  FB_DENSE_GATE = 3,    /* times sigmoid(gate[t * ld_gate + batch entry]) */
  FB_DENSE_DYT_ADD = 4, /* out (fp32) = residual + tanh(alpha acc) w + b, and, with h_out given, h_out (bf16) = tanh(alpha2 out) w2 + b2: a Dynamic
                           Tanh on a branch, the residual add, and the Dynamic Tanh that the next branch starts with */
  FB_DENSE_SWIGLU = 5,  /* as FB_DENSE_GLU, the plain unit: out = g sigmoid(g) u */
  FB_DENSE_GEGLU = 6,   /* as FB_DENSE_GLU: out = gelu(gate + gate_bias) (up + up_bias), GELU's tanh form */
  FB_DENSE_RELU2 = 7    /* out = max(v, 0)^2 */
};
typedef struct {
  int kind;
  int64_t act_cols;
  float limit, slope;
  const float* gate;
  int64_t ld_gate;
  const float* residual;
  int64_t ld_residual;
  const float *alpha, *w, *b; /* alpha: one number on the device; w, b: [N] */
  void* h_out;
  int64_t ld_h;
  const float *alpha2, *w2, *b2;
  const float *gate_bias, *up_bias; /* GEGLU: [N / 2] each, or null */
  const float* row_scale;           /* GLU, SWIGLU, RELU2: row t's sums times row_scale[t] before the unit (a weight on its input), or null */
} fb_dense_epilogue;
/* batch independent matmuls: x, W and out move on by x_batch, w_batch and out_batch elements an entry (x_batch 0: all take the
 * same rows).  ldx, ldw, x_batch, w_batch multiples of 8 elements, x and W 16-byte aligned, K a multiple of 8 (GLU: N / 2 a
 * multiple of 16); fb_dense_supports says whether a call qualifies.  settled: W was complete before the kernel launched
 * before this one (loaded weights): its first tiles are then fetched while that kernel drains. */
int fb_dense_supports(const void* x, int64_t ldx, int64_t x_batch, const void* W, int64_t ldw, int64_t w_batch, int64_t K, int64_t N, int kind);
int fb_dense(const void* x, int64_t M, int64_t K, int64_t ldx, int64_t x_batch, const void* W, int64_t N, int64_t ldw, int64_t w_batch, int64_t batch,
             void* out, int out_dtype, int64_t ldo, int64_t out_batch, const fb_dense_epilogue* epilogue_host, int settled, void* stream);

/* ---- a mixture of experts with bf16 or fp32 weights ------------------------------------------------------ */

typedef struct {
  int n, k;          /* router outputs, choices a token */
  int identity;      /* the last so many outputs stand for experts that give back their input: they have no rows */
  const float* bias; /* [n] or null: joins what the choice goes by and, unless scored, the weights */
  int scored;        /* 0: choices by logit + bias, weights the softmax of the chosen; 1: scores = softmax of all logits, choices by
                        score + bias, weights the chosen scores over their sum (+ 1e-20); 2: likewise, scores = sigmoid of each logit */
  float scale;       /* the weights times this */
  int as_scored;     /* the weights are the chosen scores themselves, not over their sum */
} fb_router;
/* Each token's k largest of its router's n outputs (fp32 logits; the lower column first among equals), their weights, and
 * where each choice's row goes (slots, both [T, k]; -1: an identity expert's) in rows of whole tiles of `tile` (a multiple of 16):
 *   shared_rows   a tile a touched expert, holding all the tokens (T <= tile): the choice's row is the token's in its expert's tile
 *   otherwise     each expert's choices in tiles of their own
 * tile_expert[tiles, 3]: each tile's expert, ascending (past those used: the number of experts with rows), that expert's first tile and its number
 * of tiles; live[0]: how many are used; tiles = fb_route_tiles(...) of the experts with rows, the most there can be.  ids [T, k]: the choices.
 * row_weights (or null): each choice's weight once more, at its row (rows that are no choice's are left alone). */
int64_t fb_route_tiles(int64_t T, int n, int k, int tile, int shared_rows);
int fb_route(const fb_router* router_host, const float* logits, int64_t T, int64_t ld, int tile, int shared_rows, float* weights, int32_t* ids,
             int32_t* slots, int32_t* tile_expert, int32_t* live, float* row_weights, void* stream);

/* Row t of x (row_bytes bytes, rows ldx_bytes apart) into the rows slots[t, 0 .. k) of out (rows one after another): the
 * tokens' rows to their choices' places. */
int fb_spread_rows(const void* x, int64_t T, int64_t row_bytes, int64_t ldx_bytes, const int32_t* slots, int k, void* out, int64_t out_rows,
                   void* stream);

/* Rows of tiles by each tile's own matrix: rows i * tile .. of out = rows i * tile .. of x (shared_rows: x's `x_rows` rows, the
 * same for every tile) @ W[tile_expert[i, 0]]^T for the tiles i < live[0]; the other rows of out are left alone.
 * fb_dense_grouped: on the tensor cores, operands as fb_dense takes them (W [n, N, K], w_batch elements apart), epilogues
 * FB_DENSE_NONE, FB_DENSE_GLU, FB_DENSE_SWIGLU and FB_DENSE_RELU2 (row_scale: one a row of out).  fb_grouped_matmul: any sizes, bf16 or
 * fp32, W by strides (matrix, row of K, column); row_scale (or null): each row of the result times its own. */
int fb_dense_grouped(const void* x, int64_t x_rows, int64_t K, int64_t ldx, int shared_rows, const void* W, int64_t N, int64_t ldw, int64_t w_batch,
                     int n, const int32_t* tile_expert, const int32_t* live, int64_t tiles, int tile, void* out, int out_dtype, int64_t ldo,
                     const fb_dense_epilogue* epilogue_host, void* stream);
int fb_grouped_matmul(int x_dtype, const void* x, int64_t x_rows, int64_t ldx, int shared_rows, int w_dtype, const void* W, const int64_t* w_strides_host, int n,
                      int64_t K, int64_t N, const int32_t* tile_expert, const int32_t* live, int64_t tiles, int tile, const float* row_scale, int out_dtype, void* out,
                      int64_t ldo, void* stream);

/* Tensor.matmul(index=) (ferrite/tensor.py:450-460; ferrite/compiler.py:704-706): a mixture of experts' matmul.  W is
 * a batch of n_experts packed [K, N] matrices fb_packed_bytes(fmt, K, N) apart; index[slot] (int32, read on the
 * device, so a replayed step follows its tokens' choices) picks one for each of n_slots slots, and a slot that picks
 * none (index >= n_experts) gives zeros with nothing read.  x: [M <= 128, K] per slot, x_slot_rows rows apart (0: every
 * slot multiplies the same x).  Prologue / epilogue as fb_linear; row_scale_bf16 (optional, [n_slots, M]) multiplies
 * each result row after the epilogue: the experts' weights (models/llama.py:322-324).
 *   sum_slots = 0: one result per slot, out + slot * out_slot_stride elements (what ferrite's batch of entries is);
 *   sum_slots = 1: x is [M, n_slots * K] (slot s's activations in columns s*K..) and the slots' matmuls are summed
 *                  into one [M, N] result in the accumulators: the experts' down projections and their sum over
 *                  the entries (llama.py:324 `.sum(0)`) in one kernel. */
int fb_linear_indexed(int fmt, const void* x, int64_t M, int64_t K, int64_t ldx, int64_t x_slot_rows, const void* W, int64_t N,
                      int n_experts, const int32_t* index, int n_slots, int sum_slots, void* out, int out_dtype, int64_t ldo,
                      int64_t out_slot_stride, const void* norm_w, float eps, int epilogue, const void* residual, int64_t ldr,
                      const void* row_scale_bf16, void* workspace, size_t workspace_bytes, void* stream);

/* ---- the rest of a decode step ------------------------------------------------------------------------- */

/* out[i, :] = table[ids[i], :]: Tensor.gather, the embedding lookup (ferrite/tensor.py:116-126,
 * ferrite/compiler.py:1574-1580).  ids are read on the device (an id outside the table is clamped into it); rows of
 * row_bytes bytes (even; whole 16-byte pieces at 16-byte aligned addresses go 16 bytes at a time). */
int fb_gather_rows(const void* table, int64_t table_rows, int64_t row_bytes, const int32_t* ids, int64_t n, void* out,
                   void* stream);

/* dst[b, ids[i], :] = src[b, i, :] for every matrix b: Tensor.put, gather's inverse (ferrite/tensor.py:128-140,
 * ferrite/compiler.py:1638-1650); of rows put at the same place the later one stays.  Strides in elements. */
int fb_put_rows(void* dst, int64_t ds0, int64_t ds1, int64_t ds2, const void* src, int64_t ss0, int64_t ss1, int64_t ss2,
                const int32_t* ids, int64_t batch, int64_t n, int64_t cols, int64_t dst_rows, int elem_bytes, void* stream);

/* After the fused qkv matmul (models/llama.py:111-128): per head optional RMSNorm of q and k heads by
 * qk_norm[(H+KV)*hd] (Qwen3, llama.py:121-123), RoPE in Hugging Face's half-rotation form with bf16 tables
 * (llama.py:92-93, 351-368), then q heads -> q_out[T, H*hd] and the k and v heads into the cache rows
 * (Tensor.put, ferrite/tensor.py:128-140; ferrite/compiler.py:1638-1650): cache[(k heads, v heads)][rows[t]][:],
 * cache laid out [2*KV, cache_rows, hd] as models/llama.py:506-514.  cos / sin: [places, table_cols] with
 * table_cols = hd (one head's table) or (H + 2*KV)*hd (ferrite's, v's columns 1 and 0).  places[t] picks the
 * table row (clamped into the table's table_rows rows), rows[t] the cache row (place + the sequence's first row,
 * llama.py:443-445; a row outside 0 .. cache_rows-1 is not written: ferrite checks neither, nothing here reads or
 * writes outside what it was given).  cache_head_stride: elements
 * from one head's rows to the next's (cache_rows * hd, or more when the cache is one sequence's part of a larger one,
 * models/llama.py:520-526). */
int fb_rope_kv_write(const void* qkv, int64_t T, int64_t ld_qkv, int H, int KV, int hd, const void* cos, const void* sin,
                     int64_t table_cols, int64_t table_rows, const int32_t* places, const int32_t* rows, const void* qk_norm, float eps,
                     void* q_out, int64_t ld_q, void* cache, int64_t cache_rows, int64_t cache_head_stride, void* stream);

/* softmax(q k^T / sqrt(hd) + mask) v over the bf16 KV cache for one token per sequence: Tensor.attend
 * (ferrite/tensor.py:487-516, ferrite/compiler.py:1147-1170) as models/llama.py:129-146 uses it.  Token t reads
 * cache rows base[t] .. base[t] + place[t] of its kv head (with window > 0 only the last `window` of them);
 * its H/KV query heads share every key row read.  max_keys: an upper bound of place[t] + 1 (it sizes the split
 * of the keys across CTAs, flash-decoding; ferrite's `parts`).  hd is 64 or 128; H/KV <= 16.
 * workspace: fb_decode_attention_workspace_bytes(...) bytes (partial sums of the key splits). */
size_t fb_decode_attention_workspace_bytes(int64_t T, int H, int KV, int hd, int64_t max_keys);
int fb_decode_attention(const void* q, int64_t T, int64_t ld_q, int H, int KV, int hd, const void* cache, int64_t cache_rows,
                        int64_t cache_head_stride, const int32_t* base, const int32_t* place, int64_t max_keys, int window, void* out, int64_t ld_o,
                        void* workspace, size_t workspace_bytes, void* stream);

/* The same two calls over a block-float KV cache (a cache in bfp8 or bfp4: models/llama.py:80,127-128; Tensor.put into a
 * block-float tensor, ferrite/compiler.py:1648-1662; pinned by test/test_sim.py:2081-2107): cache_packed holds 2 KV packed
 * matrices [cache_rows, hd] (fb_packed_bytes each), the keys' heads then the values'.  fb_rope_kv_write_packed rounds
 * each run of 16 of a new row exactly as fb_quantize does; fb_decode_attention_packed unpacks the rows it reads to the
 * same bf16 values a bf16 cache would hold and then computes what fb_decode_attention computes, bit for bit.
 * base[t] (a sequence's first cache row) must be a multiple of 64: a sequence's rows start a packed unit. */
int fb_rope_kv_write_packed(int cache_fmt, const void* qkv, int64_t T, int64_t ld_qkv, int H, int KV, int hd, const void* cos, const void* sin,
                            int64_t table_cols, int64_t table_rows, const int32_t* places, const int32_t* rows, const void* qk_norm, float eps, void* q_out,
                            int64_t ld_q, void* cache_packed, int64_t cache_rows, void* stream);
int fb_decode_attention_packed(int cache_fmt, const void* q, int64_t T, int64_t ld_q, int H, int KV, int hd, const void* cache_packed,
                               int64_t cache_rows, const int32_t* base, const int32_t* place, int64_t max_keys, int window, void* out,
                               int64_t ld_o, void* workspace, size_t workspace_bytes, void* stream);

/* The same attention for a chunk of ONE sequence's prompt (models/llama.py:498-504, forward over a prompt's tokens at
 * once): T tokens at places[t], their keys and values already in the cache rows first_row + place, each token seeing
 * the sequence's keys 0 .. place[t].  A query head's tokens are taken 16 to a CTA, so a key row is read once per 16
 * tokens of a head.  cache_fmt: FB_BF16 (cache as fb_decode_attention takes it) or FB_BFP8 / FB_BFP4 (as
 * fb_decode_attention_packed; first_row a multiple of 64).  max_keys: an upper bound of place[t] + 1. */
size_t fb_prefill_attention_workspace_bytes(int64_t T, int H, int hd, int64_t max_keys);
int fb_prefill_attention(int cache_fmt, const void* q, int64_t T, int64_t ld_q, int H, int KV, int hd, const void* cache, int64_t cache_rows,
                         int64_t cache_head_stride, int64_t first_row, const int32_t* places, int64_t max_keys, int window, void* out,
                         int64_t ld_o, void* workspace, size_t workspace_bytes, void* stream);

/* fb_decode_attention for callers that cannot provide a workspace and must not have one allocated for them (a
 * process whose own pool owns all device memory, a binding with no way to hold a scratch buffer).  It has no
 * counterpart in the reference.  The partial sums of the key splits go into an array built into the library
 * (fb_decode_attention_static_max_bytes() bytes of every GPU that loads it, from load to exit); a call that would
 * need more is refused with FB_ERR_ARG and a message.  No memory is allocated or freed by this call, ever.
 * The first call on a device looks up the array's device address: make that call outside any stream capture.
 * All calls on a device share the array and it keeps the last call's contents; nothing in it needs clearing, but
 * calls that overlap on the GPU (different streams) race on it: keep them on one stream. */
size_t fb_decode_attention_static_max_bytes(void);
int fb_decode_attention_static(const void* q, int64_t T, int64_t ld_q, int H, int KV, int hd, const void* cache, int64_t cache_rows,
                               int64_t cache_head_stride, const int32_t* base, const int32_t* place, int64_t max_keys, int window,
                               void* out, int64_t ld_o, void* stream);

/* The same kernel in ferrite's general form, Tensor.attend (ferrite/tensor.py:487-516): `entries` batch entries of
 * `rows` query rows [rows, hd] (strides in elements), every kv_rep consecutive entries reading one key and one value
 * matrix [keys, hd] (a repeat_interleave read in place, ferrite/tensor.py:210-217), and an int32 place per row
 * (place_row_stride 0: one place for all rows of an entry; place_entry_stride 0: one column of places for all
 * entries): a row sees keys 0..place (the last `window` of them).  Scores are scaled by `scale`.  out: [entries, rows, hd]. */
size_t fb_attend_workspace_bytes(int64_t entries, int64_t rows, int hd, int64_t max_keys);
int fb_attend(const void* q, int64_t entries, int64_t rows, int hd, int64_t q_entry_stride, int64_t q_row_stride, const void* k,
              const void* v, int64_t kv_entry_stride, int64_t kv_rep, int64_t keys, const int32_t* places,
              int64_t place_entry_stride, int64_t place_row_stride, int window, float scale, void* out, void* workspace,
              size_t workspace_bytes, void* stream);

/* x * rsqrt(mean(x^2) + eps) * w, row by row (models/llama.py:82-85), bf16 in and out */
int fb_rmsnorm(const void* x, int64_t rows, int64_t cols, int64_t ldx, const void* w, float eps, void* out, int64_t ldo,
               void* stream);

/* greedy pick: each row's first largest fp32 logit (what models/llama.py:787-795 does on the host with argmax);
 * out_value (optional): the maxima, for picking across vocabulary shards */
int fb_argmax(const void* logits_f32, int64_t rows, int64_t cols, int64_t ld, int32_t* out, float* out_value, void* stream);

/* ---- the mixture-of-experts router (models/llama.py:277-292) ------------------------------------------- */

/* Tensor.topk (ferrite/tensor.py:373-388, ferrite/compiler.py:1716-1731): each row's k <= 64 largest, largest first,
 * the lower column first among equals, -0 equal to 0, compared exactly as stored (dtype FB_BF16 or FB_FP32): the
 * order of numpy's stable argsort (models/llama.py:27).  values (x's dtype) and ids: [rows, k] with row stride ldo;
 * labels (optional, shaped like x): what to report instead of a pick's column.  softmax_weights_bf16 (optional,
 * [rows, k]): the softmax of each row's picked values, the experts' weights (llama.py:287-288). */
int fb_topk(int dtype, const void* x, int64_t rows, int64_t cols, int64_t ldx, int k, const int32_t* labels, void* values,
            int32_t* ids, void* softmax_weights_bf16, int64_t ldo, void* stream);

/* Tensor.touched (ferrite/tensor.py:403-416, ferrite/compiler.py:1898-1905): from ids and bf16 weights [rows, k]
 * (experts below n), experts[min(rows*k, n)]: those some row picks by a weight that is not 0, ascending, then n
 * ("none"); out_bf16[entry, row]: the row's weight for that entry's expert, 0 where it did not pick it.
 * first (0 for the reference's behaviour): experts are counted from it - a rank holding experts first .. first+n-1 of
 * a mixture spread over several GPUs lists only those, numbered from 0, and ignores the picks of other ranks' experts. */
int fb_touched(const int32_t* ids, const void* weights_bf16, int64_t rows, int k, int n, int first, int32_t* experts, void* out_bf16,
               void* stream);

/* Tensor.group (ferrite/tensor.py:389-402, ferrite/compiler.py:1842-1896): a mixture's tokens grouped by expert, from
 * int32 choices [rows, k] (values below n; others are left out).  With t = ceil(rows*k / 32) + min(n, rows*k) tiles of
 * 32 slots and rp = rows rounded up to 32:  order[32 t]: the row each slot holds (0 for none), each value's choices a
 * run of whole tiles, in the choices' own order;  tiles[t]: each tile's value (n past those used: "none" to a matmul
 * that picks by them);  places[k * rp]: run j holds, for each row, the slot of its choice j.  One kernel. */
int fb_group(const int32_t* ids, int64_t rows, int k, int n, int32_t* order, int32_t* tiles, int32_t* places, void* stream);

/* ---- the general operator surface (ferrite/tensor.py:292-372, 443-485), for expressions that are not one of the
 * fused kernels above.  Strides are in elements for (batch, row, col); a stride of 0 broadcasts.  *_host arguments
 * are host arrays read during the call. */

/* One fused elementwise expression (ferrite fuses a tree into one kernel, ferrite/compiler.py:699-738).  The
 * expression is a postfix program of n_ops (op, arg) pairs: op 0 pushes input `arg`, op 1 pushes consts_host[position];
 * 10.. are binary (add sub mul max cmplt cmpne keep drop div min), 30.. unary (exp log sin cos sqrt recip relu exp2
 * log2 round-to-bf16 trunc neg tanh).  Computed in fp32, rounded once at the store. */
int fb_elementwise(int n_ops, const int32_t* program_host, const float* consts_host, int n_inputs, const void* const* inputs_host,
                   const int64_t* strides_host, const int32_t* dtypes_host, void* out, const int64_t* out_strides_host,
                   int out_dtype, int64_t batch, int64_t rows, int64_t cols, void* stream);

/* sum or max along one axis, kept as 1 (Tensor.sum / Tensor.max, ferrite/tensor.py:359-368) */
int fb_reduce(int is_max, const void* in, const int64_t* in_strides_host, int in_dtype, int64_t batch, int64_t rows, int64_t cols,
              int axis, void* out, const int64_t* out_strides_host, int out_dtype, void* stream);

/* C[b] = A[b] @ B[b] for bf16 / fp32 operands by strides (a transposed B is a stride swap, a batch stride of 0
 * repeats a matrix): Tensor.matmul without a block-float B (ferrite/tensor.py:443-485); fp32 accumulation. */
int fb_matmul(const void* a, const int64_t* a_strides_host, int a_dtype, const void* b, const int64_t* b_strides_host, int b_dtype,
              void* c, const int64_t* c_strides_host, int c_dtype, int64_t batch, int64_t M, int64_t N, int64_t K, void* stream);

/* ---- attention over a cache of latents, rotation of neighbouring pairs, linear attention with decay ------- */

/* After a joint down-projection (row t of `down`: q_rank columns of the query latent, kv_rank of the key-value latent, rot
 * of the key part that all heads share): q_out[t] = RMSNorm(query latent) * q_norm (q_rank 0: a design without one), and
 * cache row rows[t] = RMSNorm(key-value latent) * kv_norm | the key part, its first `dims` columns turned pair by pair (2i,
 * 2i + 1) by places[t] * freq[i] with cos and sin times `mag`.  Norms and angles in fp32 or better; in_dtype: how `down`
 * is stored, dtype: q_out and the cache.  A row outside the cache is not written.
 * heads >= 1 (then q_rank is 0): the row begins with the queries instead, heads x (dim | rot): their first parts side by side to
 * q_out [T, heads * dim], the others, turned, to q_turned + t * ld_turned + h * turned_head. */
int fb_latent_put(int in_dtype, const void* down, int64_t T, int64_t ld, int q_rank, int kv_rank, int rot, int dims, const float* q_norm,
                  const float* kv_norm, float eps, const double* freq, float mag, const int32_t* places, const int32_t* rows, int dtype,
                  void* q_out, int64_t ld_q, int heads, int dim, void* q_turned, int64_t ld_turned, int64_t turned_head, void* cache,
                  int64_t cache_rows, void* stream);

/* The same turn for each head of x (head h of token t at x + t * x_row + h * x_head, `width` columns, the first `dims` of
 * them turned, the rest copied) into out (strides alike). */
int fb_rotate_pairs(int dtype, const void* x, int64_t T, int heads, int64_t x_row, int64_t x_head, int width, int dims, const double* freq,
                    float mag, const int32_t* places, void* out, int64_t o_row, int64_t o_head, void* stream);

/* Attention whose keys and values are one row of cache [cache_rows, rank + rot] a token, shared by all heads: head h of token t
 * has its query at q + t * ld_q + h * (rank + rot), scores are scale * (query . row), the output (out + t * ld_o + h * rank) is
 * the softmax-weighted sum of the rows' first `rank` columns.  Token t sees the rows base[t] + row0 + 0 .. last[t] (base null:
 * row0 alone), with window only the last `window` of them.  sink (fp32 [heads], or null): exp(sink[h]) joins head h's denominator
 * once, unscaled and without a value.
 * chunk: the tokens are consecutive ones of one sequence (they may share the rows they read).  max_keys: an upper bound of
 * last[t] + 1.  workspace: fb_latent_attention_workspace_bytes bytes. */
size_t fb_latent_attention_workspace_bytes(int dtype, int64_t T, int heads, int rank, int rot, int64_t max_keys, int chunk, int window);
int fb_latent_attention(int dtype, const void* q, int64_t T, int64_t ld_q, int heads, int rank, int rot, const void* cache, int64_t cache_rows,
                        const int32_t* base, int64_t row0, const int32_t* last, int64_t max_keys, int chunk, int window, float scale, const float* sink,
                        void* out, int64_t ld_o, void* workspace, size_t workspace_bytes, void* stream);

/* Linear attention with a decay per head, token after token: S = decay[h] * S + k v^T, out = S^T q, over `sequences`
 * sequences of `tokens` tokens each, one sequence's rows after the other's.  qkv row: q (heads x dim) | k (heads x dim) |
 * v (heads x vdim).  state: fp32 [heads, dim, vdim] per sequence, state_stride elements apart, read and left for the next
 * call.  A sequence whose first token stands at place 0 starts from zeros; one whose first token stands at place `dead`
 * (-1: none) has no token: its state is left alone and its output is 0. */
int fb_decay_scan(int dtype, const void* qkv, int64_t ld, int heads, int dim, int vdim, const float* decay, const int32_t* places, int dead,
                  int64_t sequences, int64_t tokens, float* state, int64_t state_stride, float* out, int64_t ld_o, void* stream);

/* The same with a decay and a step size per head and token (a state space): with d = softplus(step[t * ld_step + h] + step_bias[h]),
 * S = exp(-exp(a_log[h]) d) S + d k v^T, out = S^T q + skip[h] v.  A row of xbc is v (heads x vdim) | k (groups x dim) | q (groups x
 * dim); head h reads group h / (heads / groups).  The state, places and `dead` as above. */
int fb_selective_scan(int dtype, const void* xbc, int64_t ld, int heads, int groups, int dim, int vdim, const float* step, int64_t ld_step, const float* step_bias,
                      const float* a_log, const float* skip, const int32_t* places, int dead, int64_t sequences, int64_t tokens, float* state,
                      int64_t state_stride, float* out, int64_t ld_o, void* stream);

/* out = RMSNorm(x) * w * sigmoid(gate), or, before, RMSNorm(x silu(gate)) * w, row by row, each of a row's `parts` equal parts by its
 * own root mean square; x, w fp32, gate of gate_dtype, out of `dtype` */
int fb_gated_rmsnorm(const float* x, int64_t rows, int64_t cols, int64_t ldx, int gate_dtype, const void* gate, int64_t ld_g, int before, const float* w, float eps, int parts,
                     int dtype, void* out, int64_t ldo, void* stream);

/* ---- short convolutions over time and a gated linear recurrence ------------------------------------------- */

typedef struct {
  int64_t cols;
  int taps;
  const float* w;       /* [taps, cols]; the last row is the current token's */
  const float* bias;    /* [cols] or null: added to the sum */
  const float* in_bias; /* [cols] or null: added to what goes in */
  int silu;             /* the result goes through SiLU */
  const int32_t* places;
  int dead;             /* as fb_decay_scan's */
  int64_t sequences, tokens; /* `sequences` sequences of `tokens` rows each, in turn */
  float* state;         /* a sequence's last taps - 1 inputs (with in_bias), [taps - 1, cols], state_stride elements apart, read and left for */
  int64_t state_stride; /* the next call; taps 1: none */
} fb_conv;
/* out[t, c] = bias[c] + sum over j of w[j, c] in[t - taps + 1 + j, c], a causal convolution per column, zeros before a sequence's first
 * token; x of in_dtype, out of dtype */
int fb_short_conv(const fb_conv* conv_host, int in_dtype, const void* x, int64_t ld, int dtype, void* out, int64_t ld_o, void* stream);

typedef struct {
  int64_t width;
  int blocks;                  /* gate columns come in so many equal blocks of (r | i) */
  const float* lam;            /* [width] */
  float rate;                  /* the decay: log a = rate r softplus(lam) */
  const float* gate_bias;      /* [2 width], laid out as the gates, or null */
  const float* y_bias;         /* [width] or null */
  float scale;                 /* of the output */
  const int32_t* places;
  int dead;
  int64_t sequences, tokens;
  float* state;                /* [width] a sequence, state_stride elements apart */
  int64_t state_stride;
} fb_lru;
/* A gated linear recurrence per column: r and i sigmoids of the gates, a = exp(log a), S = a S + sqrt(1 - a^2) i u, out = scale S
 * gelu(y + y_bias), GELU's tanh form.  u and out of dtype, gates fp32 [rows, 2 width], y of y_dtype. */
int fb_lru_scan(const fb_lru* lru_host, int dtype, const void* u, int64_t ld_u, const float* gates, int64_t ld_gates, int y_dtype, const void* y, int64_t ld_y,
                void* out, int64_t ld_o, void* stream);

/* ---- grouped-query attention over rows of a key and its value, and what stands around it ------------------- */

/* out[t] = table[ids[t]] * scale + places_table[places[t]] (or the first alone) in fp32; ids and places outside are clamped */
int fb_embed(int dtype, const void* table, int64_t rows, int64_t cols, const int32_t* ids, const void* places_table, int64_t place_rows,
             const int32_t* places, int64_t T, float scale, float* out, void* stream);

typedef struct {
  int heads, kv_heads, dim, vdim; /* dim: a query's and a key's columns, vdim: a value's */
  const float* bias;              /* one a column of q | k | v, or null */
  const float *q_norm, *k_norm;   /* [dim]: RMSNorm of each head, all heads by the same weight; null: none */
  float eps;
  const void* first;              /* other values of the same tokens (kv_heads * vdim columns, stored as qkv is), or null: the value
                                     becomes (1 - share) value + share (first + first_bias) */
  int64_t ld_first;
  const float *first_bias, *share; /* share: one number on the device */
  int norm_all;                    /* the norms go over all query (key) heads together; q_norm [heads * dim], k_norm [kv_heads * dim] */
  int keys_are_values;             /* qkv has no v: the values are the keys as projected, before norm and turn (vdim = dim) */
  int turned;                      /* of each query and key head the first so many columns turn pair by pair (2i, 2i + 1) by */
  const double* freq;              /* places[t] * freq[i], cos and sin times mag */
  float mag;
  const int32_t* places;
  int taps;                        /* a short convolution over time, before norm, turn and cache: each column becomes the sum over j of */
  const float* conv;               /* conv[j, column] times its value (with its bias) taps - 1 - j tokens ago, zeros before the */
  float* state;                    /* sequence's start; conv [taps, columns of q | k | v], null: none.  state: the last taps - 1 rows of */
  int64_t state_stride;            /* each sequence, read and left for the next call, state_stride elements a sequence.  The T rows are */
  int sequences, dead;             /* `sequences` sequences' in turn; one whose first token stands at place 0 starts from zeros, one whose
                                      first token stands at place `dead` (-1: none) leaves its state alone */
  float temp_coef, temp_every;     /* queries, after their norm, times 1 + temp_coef ln(floor((places[t] + 1) / temp_every) + 1); 0: no such factor */
} fb_heads;
/* After a joint projection q (heads x dim) | k (kv_heads x dim) | v (kv_heads x vdim) (| more): biases and norms in fp32, queries
 * to q_out, and (key | value) into row rows[t] of each key head of cache [kv_heads, cache_rows, dim + vdim] (heads head_stride
 * elements apart; a row outside is not written).  in_dtype: how qkv is stored, dtype: q_out and the cache. */
int fb_heads_put(const fb_heads* heads_host, int in_dtype, const void* qkv, int64_t T, int64_t ld, const int32_t* rows, int dtype, void* q_out,
                 int64_t ld_q, void* cache, int64_t cache_rows, int64_t head_stride, void* stream);

/* Attention over such a cache: query head h reads key head h / (heads / kv_heads); token t, whose place is last[t], sees the cache
 * rows base[t] + row0 + lo .. + last[t] (base null: row0 alone), lo = 0, or, with span, the first place of its span of `span`
 * places; with window, only the last `window` of them.  softcap c > 0: a scaled score s becomes c tanh(s / c).  sink (fp32 [heads], or null): exp(sink[h]) joins head h's denominator.  key_bias (fp32 [heads], or null): no softmax,
 * a key's weight is sigmoid(score + key_bias[h]), and the result is the weighted sum as it is (then no sink).  The result times
 * out_scale.  gate (or null): the result times its sigmoid,
 * column by column.  chunk: the tokens are consecutive ones of one sequence.  max_keys: an upper bound of last[t] + 1. */
int fb_heads_attention(int dtype, const void* q, int64_t T, int64_t ld_q, int heads, int kv_heads, int dim, int vdim, const void* cache,
                       int64_t cache_rows, int64_t head_stride, const int32_t* base, int64_t row0, const int32_t* last, int64_t max_keys, int chunk,
                       int span, int window, float scale, float softcap, const float* sink, const float* key_bias, float out_scale, int gate_dtype, const void* gate, int64_t ld_g, void* out, int64_t ld_o,
                       void* stream);

typedef struct {
  const float* x; /* the residual stream [T, cols] */
  int64_t ld_x;
  const void* mixer; /* a branch's result and its scale by column (or null: 1) */
  int64_t ld_mixer;
  const float* mixer_scale;
  const void* other; /* the other branch's; a mixture adds to it the rows slots[t, j] of `chosen`, times weights[t, j] */
  int64_t ld_other;
  const float* other_scale;
  const void* chosen;
  int64_t ld_chosen;
  const int32_t* slots;
  const float* weights; /* null: each 1 */
  int k;
  float* x_out; /* x + mixer * mixer_scale + (other + chosen) * other_scale, or null */
  int64_t ld_x_out;
  const float* w; /* h = RMSNorm of that, times (w + plus); h null: none */
  float plus, eps;
  void* h;
  int64_t ld_h;
  const float* mixer_bias; /* added to the mixer's result (where there is none, in its place), one a column */
  const void* own;         /* the row of a choice with slot -1: token t's is row t */
  int64_t ld_own;
  const float* gate;       /* the branches' sum times sigmoid(gate[t * ld_gate + c] + gate_bias[c]), or null */
  int64_t ld_gate;
  const float* gate_bias;
  const float* post;       /* and then as RMSNorm by it leaves it (one a column, the same eps), or null: before it joins the stream */
} fb_branches;
/* A layer's end and the next one's start.  Branches null: not there; h without w: the sum itself.  in_dtype: mixer and other; dtype:
 * chosen, own and h. */
int fb_add_norm(const fb_branches* branches_host, int64_t T, int64_t cols, int in_dtype, int dtype, void* stream);

/* ---- several GPUs -------------------------------------------------------------------------------------- */

/* out = residual + sum over the ranks of their partials, bf16 [count], one kernel per rank reading the other ranks'
 * partials out of their memory over NVLink (plain peer loads).  No counterpart in the reference, which drives one chip
 * (ferrite/runtime.py:304-311); it stands where a tensor-parallel block all-reduces o_proj's / down_proj's / the
 * experts' partial sums and adds the residual (models/llama.py:95-109).
 * partials[r], flags[r]: HOST arrays of `world` device addresses, valid on this GPU, of rank r's partial for this call
 * site and of rank r's flag words (`world` uint32, zero before the first call); every rank passes the same buffers in
 * the same order and makes the same sequence of calls.  state: 4 uint32 of this GPU, zero before the first call
 * ([0] counts the calls; [2] holds 201 + r after a bounded wait for rank r gave up, else 0; [3]: the wait's bound in
 * clock cycles, 0 for the default of about two seconds).  The partial of a call site may be overwritten once a later
 * call has passed its wait (every rank has then finished reading it).  count: a multiple of 8.
 * All ranks add in rank order, so their results are bit-identical. */
int fb_peer_reduce_add(const void* const* partials, void* const* flags, int rank, int world, void* state, int64_t count,
                       const void* residual, void* out, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* FERRITE_B200_H */
