// Pieces of the causal convolutions over channels that several recurrent mixers run on the columns of a projection:
// 16 bytes of channels as floats, the update of a request's kept inputs, and the functions around them.
#pragma once
#include "common.cuh"

#define SS_MAX_TAPS 16

__device__ __forceinline__ float ss_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ss_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T> struct SsVec;
template <> struct SsVec<bf16> {
    static constexpr int W = 8;
    __device__ static void load(const bf16* src, float* v) {
        const uint4 raw = __ldg(reinterpret_cast<const uint4*>(src));
        const bf16* e = reinterpret_cast<const bf16*>(&raw);
#pragma unroll
        for (int i = 0; i < 8; i++) v[i] = __bfloat162float(e[i]);
    }
    __device__ static void store(bf16* dst, const float* v) {
        uint4 o;
        __nv_bfloat162 t;
        t = __floats2bfloat162_rn(v[0], v[1]); o.x = *reinterpret_cast<uint32_t*>(&t);
        t = __floats2bfloat162_rn(v[2], v[3]); o.y = *reinterpret_cast<uint32_t*>(&t);
        t = __floats2bfloat162_rn(v[4], v[5]); o.z = *reinterpret_cast<uint32_t*>(&t);
        t = __floats2bfloat162_rn(v[6], v[7]); o.w = *reinterpret_cast<uint32_t*>(&t);
        *reinterpret_cast<uint4*>(dst) = o;
    }
};
template <> struct SsVec<float> {
    static constexpr int W = 4;
    __device__ static void load(const float* src, float* v) {
        const float4 r = __ldg(reinterpret_cast<const float4*>(src));
        v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
    }
    __device__ static void store(float* dst, const float* v) { *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]); }
};

// The inputs a request keeps behind a segment of len rows: its last taps - 1, from the rows of this step and, where the
// segment is shorter than that, from what was kept before (zero for a fresh sequence).
template <typename T>
__global__ void __launch_bounds__(128)
ssm_conv_keep_kernel(const T* __restrict__ p, int ld, int conv_col, float* __restrict__ kept, size_t slot_stride,
                     const int* __restrict__ cu_rows, const int* __restrict__ seg_pos, const int* __restrict__ seg_slot, int C, int K) {
    kp_pdl_begin();
    const int seg = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int row0 = cu_rows[seg], row1 = cu_rows[seg + 1], len = row1 - row0;
    const bool fresh = seg_pos[seg] == 0;
    float* kp = kept + (size_t)seg_slot[seg] * slot_stride;
    for (int j = 0; j < K - 1; j++) {                       // ascending: index len + j is read before it is written
        const int rr = row1 - (K - 1) + j;
        float v;
        if (rr >= row0) v = to_f32(p[(size_t)rr * ld + conv_col + c]);
        else v = fresh ? 0.f : kp[(size_t)(len + j) * C + c];
        kp[(size_t)j * C + c] = v;
    }
}
