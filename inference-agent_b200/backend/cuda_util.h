// Error helpers shared by the backends: CUDA runtime and C-ABI status codes as exceptions.
#pragma once

#include <cuda_runtime.h>

#include <stdexcept>
#include <string>

#include "ingot_cuda.h"

inline void cuda_check(cudaError_t e, const char* what) {
    if (e != cudaSuccess) throw std::runtime_error(std::string("cuda: ") + what + ": " + cudaGetErrorString(e));
}
inline void ingot_check(int rc) {
    if (rc != INGOT_OK) throw std::runtime_error(ingot_last_error()[0] ? ingot_last_error() : ingot_status_string(rc));
}
