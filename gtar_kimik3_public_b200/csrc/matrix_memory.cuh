// What the kernels of the matrix memory share: where a token's numbers stand in the packed projection, and the two gates.
#pragma once

#include "common.cuh"

namespace memory {

struct Columns {
    int q, k, v, i, f;  // first column of q [H d], k [H d], v [H dv], z_i [H], z_f [H]
};

constexpr float DEN_ADD = 1e-6f;

__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }

// logsigmoid(x) = min(x, 0) - log(1 + e^-|x|)
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
    const float x = cap * tanhf(z / cap);
    return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

inline int sm_count() {
    static int sms = 0;
    if (sms == 0) {
        int device = 0;
        cudaGetDevice(&device);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
        if (sms <= 0) sms = 148;
    }
    return sms;
}

}  // namespace memory
