// fb_heads_attention on the tensor cores: keys of up to 256 columns
#include "heads_attention.cuh"

namespace fb {

int heads_attention_256(const HeadsArgs& a, cudaStream_t s) { return launch_values<256>(a, s); }

}  // namespace fb
