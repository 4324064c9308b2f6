// Rotary positions as the kernels that rotate whole rows of heads use them: which two entries of a head form a pair, and
// the pair's sine and cosine.  Angles are float32: position * inv_freq[pair]; the sine and the cosine are multiplied by
// `amplitude` (1: a plain rotation).
#pragma once
#include "common.cuh"

struct Rotation {
    const float* inv_freq;  // [dims / 2]
    int dims;               // the leading entries of a head that turn (even; 0: none)
    int interleaved;        // 0: entry i pairs with entry i + dims/2; 1: entry 2i pairs with entry 2i + 1
    float amplitude;
};

// The first and the second entry of pair i.
__device__ __forceinline__ int rotation_first(const Rotation& r, int i) { return r.interleaved ? 2 * i : i; }
__device__ __forceinline__ int rotation_second(const Rotation& r, int i) { return r.interleaved ? 2 * i + 1 : i + (r.dims >> 1); }

// cs[dims/2], sn[dims/2] (shared memory) for one position, by all threads of the block; the caller synchronises.
__device__ __forceinline__ void rotation_table(const Rotation& r, int position, float* cs, float* sn) {
    const float p = (float)position;
    for (int i = threadIdx.x; i < (r.dims >> 1); i += blockDim.x) {
        float s, c;
        sincosf(p * r.inv_freq[i], &s, &c);
        cs[i] = c * r.amplitude;
        sn[i] = s * r.amplitude;
    }
}

static inline bool rotation_ok(const Rotation& r, int dk) {
    return r.dims >= 0 && r.dims <= dk && (r.dims & 1) == 0 && (r.dims == 0 || r.inv_freq != nullptr);
}
