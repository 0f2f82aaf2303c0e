// fb_heads_attention on the tensor cores: keys of up to 128 columns
#include "heads_attention.cuh"

namespace fb {

int heads_attention_128(const HeadsArgs& a, cudaStream_t s) { return launch_values<128>(a, s); }

}  // namespace fb
