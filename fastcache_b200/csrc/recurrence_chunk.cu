#include "hybrid.cuh"
#include <stdexcept>
namespace fc {
bool chunk_supported(int D, int V) { return false; }
void launch_gla_chunk(const StepParams&, int, cudaStream_t) { throw std::runtime_error("no chunked form"); }
void launch_delta_chunk(const StepParams&, int, cudaStream_t) { throw std::runtime_error("no chunked form"); }
}
