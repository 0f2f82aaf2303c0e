// Linear attention with a fixed decay per head: S_t = decay S_(t-1) + k_t v_t^T (fp32, a [dim, vdim] matrix a head and
// sequence), o_t = S_t^T q_t, and the gated RMSNorm that follows it.
//
//   fb_decay_scan       token after token: a decode step's one token a sequence, and prompts in fp32 or of odd sizes
//   fb_gated_rmsnorm    RMSNorm over all the heads' outputs together, times the sigmoid of a gate
#include "values.cuh"

namespace fb {

struct ScanArgs {
  const void* qkv;  // [tokens, ld]: q (heads x dim) | k (heads x dim) | v (heads x vdim)
  int64_t ld;
  int heads, dim, vdim;
  const float* decay;     // [heads]
  const int32_t* places;  // a sequence whose first token is at place 0 starts from a zero state
  int dead;               // a sequence whose first token is at this place has no token (its state stays, its output is 0); -1: none
  int64_t tokens;         // per sequence, one sequence's after the other's
  float* state;           // [sequences, heads, dim, vdim], sequences state_stride apart
  int64_t state_stride;
  float* out;  // [tokens, ld_o]
  int64_t ld_o;
};

// A CTA keeps 32 columns of one head's state of one sequence in registers: thread (group g, lane) the rows
// 16 g .. 16 g + 15 of column `lane`.  The groups' parts of an output meet in shared memory.
constexpr int SCAN_ROWS = 16;

template <typename Act>
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
  const float decay = a.decay[h];
  for (int64_t t = 0; t < a.tokens; ++t) {
    const Act* x = static_cast<const Act*>(a.qkv) + (t0 + t) * a.ld;
    float* part = parts + (t & 1) * groups * 32;
    for (int c = threadIdx.x; c < a.dim; c += blockDim.x) {
      sq[c] = value_of(x[(int64_t)h * a.dim + c]);
      sk[c] = value_of(x[((int64_t)a.heads + h) * a.dim + c]);
    }
    const float v = mine ? value_of(x[2 * (int64_t)a.heads * a.dim + (int64_t)h * a.vdim + col]) : 0.f;
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
      a.out[(t0 + t) * a.ld_o + (int64_t)h * a.vdim + col] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < SCAN_ROWS; ++i) {
    const int row = g * SCAN_ROWS + i;
    if (mine && row < a.dim) state[(int64_t)row * a.vdim + col] = S[i];
  }
}

template <typename Act>
__global__ void __launch_bounds__(256) gated_rmsnorm_kernel(const float* x, int64_t ldx, const void* gate, int64_t ld_g, const float* w, float eps,
                                                            int64_t cols, void* out, int64_t ldo) {
  griddep_launch_dependents();
  griddep_wait();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  float ss = 0.f;
  for (int64_t c = threadIdx.x; c < cols; c += blockDim.x) ss = fmaf(x[t * ldx + c], x[t * ldx + c], ss);
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)cols + eps);
  const Act* g = static_cast<const Act*>(gate) + t * ld_g;
  for (int64_t c = threadIdx.x; c < cols; c += blockDim.x)
    store_value(static_cast<Act*>(out) + t * ldo + c, x[t * ldx + c] * r * w[c] * sigmoid_f(value_of(g[c])));
}

}  // namespace fb

extern "C" int fb_decay_scan(int dtype, const void* qkv, int64_t ld, int heads, int dim, int vdim, const float* decay, const int32_t* places, int dead,
                             int64_t sequences, int64_t tokens, float* state, int64_t state_stride, float* out, int64_t ld_o, void* stream) {
  FB_REQUIRE(qkv && decay && places && state && out && sequences >= 1 && tokens >= 1 && heads >= 1 && dim >= 1 && vdim >= 1, "fb_decay_scan: null pointer or empty");
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "fb_decay_scan: bf16 or fp32");
  FB_REQUIRE(dim <= 512, "fb_decay_scan: heads of up to 512 query columns (got %d)", dim);
  FB_REQUIRE(ld >= (int64_t)heads * (2 * dim + vdim) && ld_o >= (int64_t)heads * vdim && state_stride >= (int64_t)heads * dim * vdim && sequences <= 65535 && heads <= 65535,
             "fb_decay_scan: row strides too small");
  fb::ScanArgs a{qkv, ld, heads, dim, vdim, decay, places, dead, tokens, state, state_stride, out, ld_o};
  const int groups = (dim + fb::SCAN_ROWS - 1) / fb::SCAN_ROWS;
  const dim3 grid((unsigned)fb::ceil_div(vdim, 32), (unsigned)heads, (unsigned)sequences);
  const size_t smem = (2 * (size_t)dim + 2 * groups * 32) * sizeof(float);
  if (dtype == FB_FP32) fb::decay_scan_kernel<float><<<grid, 32 * groups, smem, (cudaStream_t)stream>>>(a);
  else fb::decay_scan_kernel<uint16_t><<<grid, 32 * groups, smem, (cudaStream_t)stream>>>(a);
  return fb::launch_status("fb_decay_scan");
}

extern "C" int fb_gated_rmsnorm(const float* x, int64_t rows, int64_t cols, int64_t ldx, int dtype, const void* gate, int64_t ld_g, const float* w, float eps,
                                void* out, int64_t ldo, void* stream) {
  FB_REQUIRE(x && gate && w && out && rows >= 1 && cols >= 1 && ldx >= cols && ld_g >= cols && ldo >= cols, "fb_gated_rmsnorm: bad arguments");
  FB_REQUIRE(dtype == FB_BF16 || dtype == FB_FP32, "fb_gated_rmsnorm: bf16 or fp32");
  if (dtype == FB_FP32) fb::gated_rmsnorm_kernel<float><<<(unsigned)rows, 256, 0, (cudaStream_t)stream>>>(x, ldx, gate, ld_g, w, eps, cols, out, ldo);
  else fb::gated_rmsnorm_kernel<uint16_t><<<(unsigned)rows, 256, 0, (cudaStream_t)stream>>>(x, ldx, gate, ld_g, w, eps, cols, out, ldo);
  return fb::launch_status("fb_gated_rmsnorm");
}
