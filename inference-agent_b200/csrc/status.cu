// Error reporting and build information of the library, shared by every entry point.
#include <cstdlib>

#include "ingot_internal.cuh"

static thread_local std::string g_last_error;

void ingot_set_error(const std::string& msg) { g_last_error = msg; }

int ingot_cuda_fail(cudaError_t e, const char* what) {
    g_last_error = std::string(what) + ": " + cudaGetErrorString(e);
    return e == cudaErrorMemoryAllocation ? INGOT_ERR_NOMEM : INGOT_ERR_CUDA;
}

bool ingot_use_pdl() {
    static const bool v = getenv("INGOT_NO_PDL") == nullptr;
    return v;
}

extern "C" {

const char* ingot_status_string(int status) {
    switch (status) {
        case INGOT_OK: return "ok";
        case INGOT_ERR_INVALID: return "invalid argument";
        case INGOT_ERR_CUDA: return "CUDA call failed";
        case INGOT_ERR_UNSUPPORTED: return "unsupported shape or dtype";
        case INGOT_ERR_NOMEM: return "out of device memory";
        case INGOT_ERR_DEVICE: return "a kernel reported an error";
        default: return "unknown status";
    }
}

const char* ingot_last_error(void) { return g_last_error.c_str(); }

const char* ingot_build_arch(void) { return "sm_100a"; }

const char* ingot_build_flags(void) {
#ifdef INGOT_BOUNDS_CHECK
    return "bounds-check";
#else
    return "";
#endif
}

}  // extern "C"
