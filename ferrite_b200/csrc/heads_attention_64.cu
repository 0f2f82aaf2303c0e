// fb_heads_attention on the tensor cores: keys of up to 64 columns
#include "heads_attention.cuh"

namespace fb {

int heads_attention_64(const HeadsArgs& a, cudaStream_t s) { return launch_values<64>(a, s); }

}  // namespace fb
