#include "hybrid.cuh"
#include <stdexcept>
namespace fc {
bool head_linear_mma_supported(const SimtLinear&) { return false; }
void launch_head_linear_mma(const SimtLinear&, cudaStream_t) { throw std::runtime_error("-"); }
bool latent_decode_supported(const LatentAttn&) { return false; }
int latent_decode_splits(const LatentAttn&, int, int) { return 1; }
void launch_latent_decode(const LatentAttn&, cudaStream_t) { throw std::runtime_error("-"); }
}
