#include "hybrid.cuh"
#include <stdexcept>
namespace fc {
bool latent_prefill_supported(const LatentPrefill&) { return false; }
void launch_latent_prefill(const LatentPrefill&, cudaStream_t) { throw std::runtime_error("-"); }
}
