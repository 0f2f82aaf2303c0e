// fb_heads_attention on the tensor cores: keys of up to 192 columns
#include "heads_attention.cuh"

namespace fb {

int heads_attention_192(const HeadsArgs& a, cudaStream_t s) { return launch_values<192>(a, s); }

}  // namespace fb
