// A residual of several streams: x [rows][S][d], float32.  A sublayer reads one weighted sum of a row's streams, normed;
// behind it every stream becomes a weighted sum of all the old streams plus its share of the sublayer's output:
//   x'_b = out_b y + sum_a mix_ab x_a ,     h = w * norm(sum_b in_b x'_b)
// in one pass over the row (the y it read is cleared for whoever adds into it next; h in the storage type is what the next
// sublayer reads).  norm: a layer norm without a shift (centred: mean taken off, variance about the mean), or the RMS norm.
// All float32 with a fixed tree a row.
#include "common.cuh"

#define ST_MAX 8                 // streams
#define ST_THREADS 256

template <typename T> __device__ __forceinline__ void st_store4(T* dst, float a, float b, float c, float d);
template <> __device__ __forceinline__ void st_store4<float>(float* dst, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void st_store4<bf16>(bf16* dst, float a, float b, float c, float d) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    uint2 v;
    v.x = *reinterpret_cast<const uint32_t*>(&lo);
    v.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = v;
}

// every stream of a row starts as the row itself
__global__ void streams_enter_kernel(const float* __restrict__ e, float* __restrict__ x, size_t n, int d, int S) {
    kp_pdl_begin();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n * d; i += (size_t)gridDim.x * blockDim.x) {
        const size_t r = i / d, c = i - r * d;
        const float v = e[i];
        for (int s = 0; s < S; s++) x[(r * S + s) * d + c] = v;
    }
}

// The coefficients a row's pass needs: mix [S][S] (from, to), out [S] (with y), in [S] (null: ones)
template <int S>
struct StCoef {
    float mix[S][S], out[S], in[S];
    __device__ __forceinline__ void load(const float* m, const float* o, const float* i, bool mixing) {
#pragma unroll
        for (int a = 0; a < S; a++) {
            in[a] = i ? __ldg(i + a) : 1.f;
            out[a] = mixing ? __ldg(o + a) : 0.f;
#pragma unroll
            for (int b = 0; b < S; b++) mix[a][b] = mixing ? __ldg(m + a * S + b) : 0.f;
        }
    }
};

// Rows of any length: the streams' new values go out first and are read again (by the thread that wrote them).
template <typename T, int S>
__global__ void __launch_bounds__(ST_THREADS)
streams_rows_kernel(float* x, float* y, const float* __restrict__ mix, const float* __restrict__ outw, const float* __restrict__ inw,
                    const float* __restrict__ w, float eps, int centred, const int* __restrict__ rows, T* __restrict__ h, int d) {
    kp_pdl_begin();
    __shared__ float red[32];
    const int r = rows ? rows[blockIdx.x] : (int)blockIdx.x;
    float* xr = x + (size_t)r * S * d;
    StCoef<S> k;
    k.load(mix, outw, inw, y != nullptr);
    float sum = 0.f;
    auto read = [&](int i) {
        float u = 0.f;
#pragma unroll
        for (int t = 0; t < S; t++) u = fmaf(k.in[t], xr[(size_t)t * d + i], u);
        return u;
    };
    for (int i = threadIdx.x; i < d; i += ST_THREADS) {
        if (y) {
            float v[S];
#pragma unroll
            for (int s = 0; s < S; s++) v[s] = xr[(size_t)s * d + i];
            const float yv = y[(size_t)r * d + i];
            y[(size_t)r * d + i] = 0.f;
#pragma unroll
            for (int t = 0; t < S; t++) {
                float z = k.out[t] * yv;
#pragma unroll
                for (int s = 0; s < S; s++) z = fmaf(k.mix[s][t], v[s], z);
                xr[(size_t)t * d + i] = z;
            }
        }
        if (h) sum += read(i);
    }
    if (!h) return;
    const float mean = centred ? block_sum(sum, red) / (float)d : 0.f;
    float ss = 0.f;
    for (int i = threadIdx.x; i < d; i += ST_THREADS) {
        const float v = read(i) - mean;
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
    const float scale = 1.0f / sqrtf(ss / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += ST_THREADS) h[(size_t)blockIdx.x * d + i] = from_f32<T>((read(i) - mean) * scale * w[i]);
}

// The same for 16-byte aligned rows of at most 4 NTH PER floats (d % 4 == 0): a thread fetches what it needs of the row at once
// and keeps u in registers, so streams and y are read once and leave in 16-byte stores.  Which form runs depends on the
// row's length and the buffers' alignment alone.
template <typename T, int S, int NTH, int PER, bool MIX>
__global__ void __launch_bounds__(NTH)
streams_rows_vec_kernel(float* x, float* y, const float* __restrict__ mix, const float* __restrict__ outw, const float* __restrict__ inw,
                        const float* __restrict__ w, float eps, int centred, const int* __restrict__ rows, T* __restrict__ h, int d) {
    kp_pdl_begin();
    __shared__ float red[32];
    const int r = !MIX && rows ? rows[blockIdx.x] : (int)blockIdx.x;
    const int n4 = d >> 2;
    float4* xr = reinterpret_cast<float4*>(x + (size_t)r * S * d);
    float4* yr = reinterpret_cast<float4*>(y + (size_t)r * d);
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 v[PER][S], yv[PER], u[PER];
#pragma unroll
    for (int j = 0; j < PER; j++) {
        const int i = threadIdx.x + j * NTH;
        const bool ok = i < n4;
#pragma unroll
        for (int s = 0; s < S; s++) v[j][s] = ok ? xr[(size_t)s * n4 + i] : zero;
        yv[j] = MIX && ok ? yr[i] : zero;
    }
    StCoef<S> k;
    k.load(mix, outw, inw, MIX);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < PER; j++) {
        const int i = threadIdx.x + j * NTH;
        u[j] = zero;
#pragma unroll
        for (int t = 0; t < S; t++) {
            float4 z = v[j][t];
            if (MIX) {
                z = make_float4(k.out[t] * yv[j].x, k.out[t] * yv[j].y, k.out[t] * yv[j].z, k.out[t] * yv[j].w);
#pragma unroll
                for (int s = 0; s < S; s++) {
                    const float m = k.mix[s][t];
                    z.x = fmaf(m, v[j][s].x, z.x); z.y = fmaf(m, v[j][s].y, z.y); z.z = fmaf(m, v[j][s].z, z.z); z.w = fmaf(m, v[j][s].w, z.w);
                }
                if (i < n4) xr[(size_t)t * n4 + i] = z;
            }
            u[j].x = fmaf(k.in[t], z.x, u[j].x); u[j].y = fmaf(k.in[t], z.y, u[j].y);
            u[j].z = fmaf(k.in[t], z.z, u[j].z); u[j].w = fmaf(k.in[t], z.w, u[j].w);
        }
        if (MIX && i < n4) yr[i] = zero;
        sum += (u[j].x + u[j].y) + (u[j].z + u[j].w);
    }
    if (!h) return;
    const float mean = centred ? block_sum(sum, red) / (float)d : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; j++) {
        if (threadIdx.x + j * NTH >= n4) continue;
        u[j].x -= mean; u[j].y -= mean; u[j].z -= mean; u[j].w -= mean;
        ss = fmaf(u[j].x, u[j].x, ss); ss = fmaf(u[j].y, u[j].y, ss); ss = fmaf(u[j].z, u[j].z, ss); ss = fmaf(u[j].w, u[j].w, ss);
    }
    ss = block_sum(ss, red);
    const float scale = 1.0f / sqrtf(ss / (float)d + eps);
#pragma unroll
    for (int j = 0; j < PER; j++) {
        const int i = threadIdx.x + j * NTH;
        if (i >= n4) continue;
        const float4 ww = __ldg(reinterpret_cast<const float4*>(w) + i);
        st_store4<T>(h + (size_t)blockIdx.x * d + 4 * i, u[j].x * scale * ww.x, u[j].y * scale * ww.y, u[j].z * scale * ww.z,
                     u[j].w * scale * ww.w);
    }
}

template <int S>
static int st_rows(float* x, float* y, const float* mix, const float* outw, const float* inw, const float* w, float eps, int centred,
                   const int* rows, void* h, int n, int d, int dtype, cudaStream_t s) {
    // (more than four streams: a thread holds one float4 of each, for rows of at most 2,048)
    constexpr bool few = S <= 4;
    const bool vec = (d & 3) == 0 && d <= (few ? 8192 : 2048) && !(((uintptr_t)x | (uintptr_t)y | (uintptr_t)w | (uintptr_t)h) & 15);
#define ST_VEC_M(NTH, PER, MIX)                                                                                              \
    KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(streams_rows_vec_kernel<T, S, NTH, PER, MIX>, dim3(n), dim3(NTH), 0, s, x, y, mix, outw, inw, w, \
                                               eps, centred, rows, (T*)h, d)))
#define ST_VEC(NTH, PER) do { if (y) ST_VEC_M(NTH, PER, true); else ST_VEC_M(NTH, PER, false); } while (0)
    if (vec) {
        if constexpr (few) {
            if (d <= 1024) ST_VEC(128, 2);
            else if (d <= 2048) ST_VEC(256, 2);
            else if (d <= 4096) ST_VEC(512, 2);
            else ST_VEC(1024, 2);
        } else {
            if (d <= 1024) ST_VEC(256, 1);
            else ST_VEC(512, 1);
        }
    } else {
        KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(streams_rows_kernel<T, S>, dim3(n), dim3(ST_THREADS), 0, s, x, y, mix, outw, inw, w, eps,
                                                   centred, rows, (T*)h, d)));
    }
#undef ST_VEC
#undef ST_VEC_M
    return kp_launch_status();
}

extern "C" {

int kp_streams_enter(const float* e, float* x, int n, int d, int S, void* stream) {
    if (n <= 0) return 0;
    if (d < 1 || S < 1) return KP_ERR_BAD_ARG;
    size_t blocks = ((size_t)n * d + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    kp_launch_pdl(streams_enter_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, e, x, (size_t)n, d, S);
    return kp_launch_status();
}

// y null: the streams stay as they are (mix and outw unused).  h null: no weighted sum is normed (inw and w unused).  rows (with
// y null): the rows of x to read.  inw null: ones.  dtype: the type of h.
int kp_streams_rows(float* x, float* y, const float* mix, const float* outw, const float* inw, const float* w, float eps, int centred,
                    const int* rows, void* h, int n, int d, int S, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (d < 1 || S < 1 || (y && (!mix || !outw || rows)) || (!y && !h) || (h && !w)) return KP_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    switch (S) {
        case 1: return st_rows<1>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        case 2: return st_rows<2>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        case 3: return st_rows<3>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        case 4: return st_rows<4>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        case 5: return st_rows<5>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        case 6: return st_rows<6>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        case 7: return st_rows<7>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        case 8: return st_rows<8>(x, y, mix, outw, inw, w, eps, centred, rows, h, n, d, dtype, s);
        default: return KP_ERR_UNSUPPORTED;
    }
}

}  // extern "C"
