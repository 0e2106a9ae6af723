// Fused per-head RMSNorm of q and k, rotary position encoding, and the write
// of k and v into the paged cache.
//
// Input rows hold [q: H*hd | k: G*hd | v: G*hd].  For each q and k head
//   x <- (x * rsqrt(mean(x^2) + eps)) * w          (src/backend/cpu/scalar/quants.c:1521-1531)
// then, for j < rot/2 with c,s = cos,sin(pos * theta^(-2j/rot)) from a table
// built in double precision (src/compute.c:22-65):
//   neox pairing (j, j + rot/2), interleaved pairing (2j, 2j+1):
//   (a, b) <- (a c - b s, a s + b c)               (src/backend/cpu/quants.h:395-409)
// q goes to q_out; k and v go to the page and offset given by slot_map
// (cache layout [page][K|V][G][page_size][hd]; src/backend/cpu/common.c:1603-1694
// stores the same rows at [layer][kv head][pos][hd]).
// Norm (w == nullptr) and rotation (cos_tab == nullptr) can each be left out.
// With q_out == nullptr, q and k are normed/rotated in place and nothing is
// written to the cache (for a position encoding applied between two calls).
// `norm_dim` (<= hd): the number the norm's mean is taken over, for heads stored wider than they are with
// zeros behind their own columns.  A query temperature (temp_every > 0): the query heads of the row at position
// p leave multiplied by 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1), computed in float32.
// `norm_after`: instead of the norm in front of the rotation q and k are divided by their root mean square behind it
// (no weight).
#include "common.cuh"

#define KP_MAX_HEAD_DIM 256

__device__ __forceinline__ float kp_query_temperature(int pos, float coef, float every) {
    return 1.0f + coef * logf(floorf((float)(pos + 1) / every) + 1.0f);
}

template <typename T>
__global__ void __launch_bounds__(128)
qk_norm_rope_kv_kernel(const T* qkv, int ld, const float* __restrict__ q_w,
                       const float* __restrict__ k_w, float eps, const float* __restrict__ cos_tab,
                       const float* __restrict__ sin_tab, int rot, int interleaved,
                       const int* __restrict__ positions, const int* __restrict__ slot_map,
                       T* q_out, int ldq, T* __restrict__ cache, int page_size,
                       int H, int G, int hd, int write_kv, int v_col, int norm_dim, float temp_coef, float temp_every,
                       int norm_after) {
    kp_pdl_begin();
    __shared__ float buf[4][KP_MAX_HEAD_DIM];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x * 4 + warp;          // 0..H-1 q, H..H+G-1 k, H+G..H+2G-1 v
    const int row = blockIdx.y;
    if (head >= H + 2 * G) return;
    const int kind = head < H ? 0 : (head < H + G ? 1 : 2);
    const bool in_place = q_out == nullptr;            // norm/rotate q and k where they are; no cache write
    if (kind != 0 && !write_kv && !(in_place && kind == 1)) return;
    // (the values start at column v_col of the row: behind the keys, or at the keys themselves for a design
    // whose values are its key projections, taken here before the key's norm and rotation)
    const T* src = qkv + (size_t)row * ld + (kind == 2 ? (size_t)v_col + (size_t)(head - H - G) * hd : (size_t)head * hd);
    float* x = buf[warp];

    float ss = 0.f;
    for (int i = lane; i < hd; i += 32) {
        const float v = to_f32(src[i]);
        x[i] = v;
        ss = fmaf(v, v, ss);
    }
    const float* w = kind == 0 ? q_w : (kind == 1 ? k_w : nullptr);
    if (w) {
        ss = warp_sum(ss);
        const float scale = 1.0f / sqrtf(ss / (float)norm_dim + eps);
        for (int i = lane; i < hd; i += 32) x[i] = (x[i] * scale) * w[i];
    }
    __syncwarp();
    if (kind != 2 && cos_tab) {
        const int half = rot >> 1;
        const size_t tb = (size_t)positions[row] * half;
        for (int j = lane; j < half; j += 32) {
            const int ia = interleaved ? 2 * j : j;
            const int ib = interleaved ? 2 * j + 1 : j + half;
            const float c = cos_tab[tb + j], s = sin_tab[tb + j];
            const float a = x[ia], b = x[ib];
            x[ia] = a * c - b * s;
            x[ib] = a * s + b * c;
        }
        __syncwarp();
    }
    if (norm_after && kind != 2) {
        float sq = 0.f;
        for (int i = lane; i < hd; i += 32) sq = fmaf(x[i], x[i], sq);
        sq = warp_sum(sq);
        const float scale = 1.0f / sqrtf(sq / (float)norm_dim + eps);
        for (int i = lane; i < hd; i += 32) x[i] *= scale;
    }
    if (kind == 0 && temp_every > 0.f) {
        const float tq = kp_query_temperature(positions[row], temp_coef, temp_every);
        for (int i = lane; i < hd; i += 32) x[i] *= tq;
    }
    T* dst;
    if (in_place) {
        dst = const_cast<T*>(src);
    } else if (kind == 0) {
        dst = q_out + (size_t)row * ldq + (size_t)head * hd;
    } else {
        const int slot = slot_map[row];
        if (slot < 0) return;
        const int page = slot / page_size, off = slot % page_size;
        const int g = kind == 1 ? head - H : head - H - G;
        dst = cache + ((((size_t)page * 2 + (kind - 1)) * G + g) * page_size + off) * hd;
    }
    for (int i = lane; i < hd; i += 32) dst[i] = from_f32<T>(x[i]);
}

// The same for bfloat16 with head size 64 or 128, NeoX rotation of the first `rot` dimensions (rot / 16 a power
// of two; or none) and 16-byte aligned rows: a thread holds 8 consecutive elements of a head (one 16-byte load
// and one 16-byte store), hd / 8 lanes share a head; the sum of squares and the rotation partner (element
// i + rot/2: the lane rot/16 further on) come by warp shuffles.  Same arithmetic in the same order as the
// general kernel.
template <int HD>
__global__ void __launch_bounds__(128)
qk_norm_rope_kv_vec_kernel(const bf16* __restrict__ qkv, int ld, const float* __restrict__ q_w,
                           const float* __restrict__ k_w, float eps, const float* __restrict__ cos_tab,
                           const float* __restrict__ sin_tab, const int* __restrict__ positions,
                           const int* __restrict__ slot_map, bf16* __restrict__ q_out, int ldq,
                           bf16* __restrict__ cache, int page_size, int H, int G, int write_kv, int v_col, int rot,
                           int norm_dim, float temp_coef, float temp_every, int norm_after) {
    kp_pdl_begin_early();
    constexpr int L = HD / 8;                          // lanes a head
    constexpr int HPB = 128 / L;                       // heads a block
    const int lane_in = threadIdx.x % L;
    const int head = blockIdx.x * HPB + threadIdx.x / L;
    const int row = blockIdx.y;
    const bool live = head < H + 2 * G;
    const int hh = live ? head : 0;
    const int kind = hh < H ? 0 : (hh < H + G ? 1 : 2);
    const size_t col = kind == 2 ? (size_t)v_col + (size_t)(hh - H - G) * HD : (size_t)hh * HD;
    const uint4 raw = *reinterpret_cast<const uint4*>(qkv + (size_t)row * ld + col + lane_in * 8);
    float x[8];
    {
        const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; i++) { const float2 f = __bfloat1622float2(p2[i]); x[2 * i] = f.x; x[2 * i + 1] = f.y; }
    }
    const float* w = kind == 0 ? q_w : (kind == 1 ? k_w : nullptr);
    if (w) {                                            // (uniform over the lanes of a head)
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) ss = fmaf(x[i], x[i], ss);
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float scale = 1.0f / sqrtf(ss / (float)norm_dim + eps);
        const float4 w0 = __ldg(reinterpret_cast<const float4*>(w + lane_in * 8));
        const float4 w1 = __ldg(reinterpret_cast<const float4*>(w + lane_in * 8) + 1);
        const float ww[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
        for (int i = 0; i < 8; i++) x[i] = (x[i] * scale) * ww[i];
    }
    if (cos_tab != nullptr) {                          // every lane takes part in the shuffles
        const int rl = rot >> 4;                       // lanes that hold one half of the rotated dimensions
        const bool lower = lane_in < rl;               // holds the `a` of its pairs; the partner holds `b`
        const bool rotated = lane_in < 2 * rl;         // (the lanes behind pass their elements on unchanged)
        const size_t tb = (size_t)positions[row] * (rot >> 1) + (size_t)(lane_in % rl) * 8;
        const float4 c0 = __ldg(reinterpret_cast<const float4*>(cos_tab + tb)), c1 = __ldg(reinterpret_cast<const float4*>(cos_tab + tb) + 1);
        const float4 s0 = __ldg(reinterpret_cast<const float4*>(sin_tab + tb)), s1 = __ldg(reinterpret_cast<const float4*>(sin_tab + tb) + 1);
        const float cc[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
        const float sn[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const float other = __shfl_xor_sync(0xffffffffu, x[i], rl);
            if (kind != 2 && rotated) x[i] = lower ? x[i] * cc[i] - other * sn[i] : other * sn[i] + x[i] * cc[i];
        }
    }
    if (norm_after) {                                  // (every lane takes part in the shuffles)
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) ss = fmaf(x[i], x[i], ss);
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float scale = 1.0f / sqrtf(ss / (float)norm_dim + eps);
        if (kind != 2) {
#pragma unroll
            for (int i = 0; i < 8; i++) x[i] *= scale;
        }
    }
    if (!live || (kind != 0 && !write_kv)) return;
    if (kind == 0 && temp_every > 0.f) {
        const float tq = kp_query_temperature(positions[row], temp_coef, temp_every);
#pragma unroll
        for (int i = 0; i < 8; i++) x[i] *= tq;
    }
    uint4 o;
    {
        __nv_bfloat162* p2 = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int i = 0; i < 4; i++) p2[i] = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
    }
    bf16* dst;
    if (kind == 0) {
        dst = q_out + (size_t)row * ldq + (size_t)head * HD;
    } else {
        const int slot = slot_map[row];
        if (slot < 0) return;
        const int page = slot / page_size, off = slot % page_size;
        const int g = kind == 1 ? head - H : head - H - G;
        dst = cache + ((((size_t)page * 2 + (kind - 1)) * G + g) * page_size + off) * HD;
    }
    *reinterpret_cast<uint4*>(dst + lane_in * 8) = o;
}

extern "C" int kp_qk_norm_rope_kv_after(const void* qkv, int ld, const float* q_w, const float* k_w, float eps,
                                        const float* cos_tab, const float* sin_tab, int rot, int interleaved,
                                        const int* positions, const int* slot_map, void* q_out, int ldq, void* cache,
                                        int page_size, int n, int H, int G, int hd, int write_kv, int v_col, int norm_dim,
                                        float temp_coef, float temp_every, int norm_after, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (norm_after && (q_w || k_w || q_out == nullptr)) return KP_ERR_BAD_ARG;
    if (norm_dim <= 0) norm_dim = hd;
    if (norm_dim > hd || temp_every < 0.f) return KP_ERR_BAD_ARG;
    if (v_col < 0) v_col = (H + G) * hd;
    if (hd < 2 || hd > KP_MAX_HEAD_DIM || (hd & 1)) return KP_ERR_UNSUPPORTED;
    if (cos_tab && (rot < 2 || rot > hd || (rot & 1))) return KP_ERR_BAD_ARG;
    if (n > 65535) return KP_ERR_UNSUPPORTED;
    // the 16-byte form: bfloat16, head size 64 or 128, NeoX rotation of 16, 32, 64 or 128 dimensions or none, aligned rows
    const bool rot_ok = !cos_tab || (!interleaved && (rot == 16 || rot == 32 || rot == 64 || rot == 128) && rot <= hd);
    if (!cos_tab) rot = hd;
    if (dtype == KP_DTYPE_BF16 && (hd == 64 || hd == 128) && q_out != nullptr && rot_ok &&
        (ld % 8 == 0) && (ldq % 8 == 0) && (v_col % 8 == 0) && !((uintptr_t)qkv & 15) && !((uintptr_t)q_out & 15) && !((uintptr_t)cache & 15) &&
        (!q_w || !((uintptr_t)q_w & 15)) && (!k_w || !((uintptr_t)k_w & 15)) &&
        (!cos_tab || (!((uintptr_t)cos_tab & 15) && !((uintptr_t)sin_tab & 15)))) {
        const int hpb = 128 / (hd / 8);
        dim3 vgrid((H + 2 * G + hpb - 1) / hpb, n);
        if (hd == 64)
            kp_launch_pdl(qk_norm_rope_kv_vec_kernel<64>, dim3(vgrid), dim3(128), 0, (cudaStream_t)stream, (const bf16*)qkv, ld, q_w,
                          k_w, eps, cos_tab, sin_tab, positions, slot_map, (bf16*)q_out, ldq, (bf16*)cache, page_size, H, G, write_kv, v_col, rot,
                          norm_dim, temp_coef, temp_every, norm_after);
        else
            kp_launch_pdl(qk_norm_rope_kv_vec_kernel<128>, dim3(vgrid), dim3(128), 0, (cudaStream_t)stream, (const bf16*)qkv, ld, q_w,
                          k_w, eps, cos_tab, sin_tab, positions, slot_map, (bf16*)q_out, ldq, (bf16*)cache, page_size, H, G, write_kv, v_col, rot,
                          norm_dim, temp_coef, temp_every, norm_after);
        return kp_launch_status();
    }
    dim3 grid((H + 2 * G + 3) / 4, n);
    KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(qk_norm_rope_kv_kernel<T>, dim3(grid), dim3(128), 0, (cudaStream_t)stream, 
        (const T*)qkv, ld, q_w, k_w, eps, cos_tab, sin_tab, rot, interleaved, positions, slot_map, (T*)q_out, ldq,
        (T*)cache, page_size, H, G, hd, write_kv, v_col, norm_dim, temp_coef, temp_every, norm_after)));
    return kp_launch_status();
}

extern "C" int kp_qk_norm_rope_kv_temp(const void* qkv, int ld, const float* q_w, const float* k_w, float eps,
                                       const float* cos_tab, const float* sin_tab, int rot, int interleaved,
                                       const int* positions, const int* slot_map, void* q_out, int ldq, void* cache,
                                       int page_size, int n, int H, int G, int hd, int write_kv, int v_col, int norm_dim,
                                       float temp_coef, float temp_every, int dtype, void* stream) {
    return kp_qk_norm_rope_kv_after(qkv, ld, q_w, k_w, eps, cos_tab, sin_tab, rot, interleaved, positions, slot_map, q_out, ldq,
                                    cache, page_size, n, H, G, hd, write_kv, v_col, norm_dim, temp_coef, temp_every, 0, dtype, stream);
}

extern "C" int kp_qk_norm_rope_kv(const void* qkv, int ld, const float* q_w, const float* k_w, float eps,
                                  const float* cos_tab, const float* sin_tab, int rot, int interleaved,
                                  const int* positions, const int* slot_map, void* q_out, int ldq, void* cache,
                                  int page_size, int n, int H, int G, int hd, int write_kv, int v_col, int dtype,
                                  void* stream) {
    return kp_qk_norm_rope_kv_temp(qkv, ld, q_w, k_w, eps, cos_tab, sin_tab, rot, interleaved, positions, slot_map, q_out, ldq,
                                   cache, page_size, n, H, G, hd, write_kv, v_col, hd, 0.f, 0.f, dtype, stream);
}

// ------------------------------------------------------------------------------------------------------------
// The norm over whole projections: q and k are RMS-normed each as one row over all their heads at once,
//   q <- q * rsqrt(sum(q^2) / count_q + eps) * w_q        (w_q as long as the projection; the same for k)
// without any rotation; q goes to q_out, k (normed) and v (as it is) to the page and offset given by slot_map.
// A head may be stored wider than it is (zero columns behind its own, as the weights' zero rows leave them), so the
// counts of the means are arguments of their own.  write_kv == 0: a layer that reads another layer's keys and values
// norms its queries only.
template <typename T>
__global__ void __launch_bounds__(256)
qk_rownorm_kv_kernel(const T* __restrict__ qkv, int ld, int k_col, int v_col, const float* __restrict__ q_w,
                     const float* __restrict__ k_w, float eps, float count_q, float count_k, const int* __restrict__ slot_map,
                     T* __restrict__ q_out, int ldq, T* __restrict__ cache, int page_size, int H, int G, int hd, int write_kv) {
    kp_pdl_begin();
    __shared__ float red[32];
    const int row = blockIdx.x;
    const T* src = qkv + (size_t)row * ld;
    const int nq = H * hd, nk = G * hd;
    float ss = 0.f;
    for (int i = threadIdx.x; i < nq; i += blockDim.x) {
        const float v = to_f32(src[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, red);
    const float sq = 1.0f / sqrtf(ss / count_q + eps);
    for (int i = threadIdx.x; i < nq; i += blockDim.x)
        q_out[(size_t)row * ldq + i] = from_f32<T>((to_f32(src[i]) * sq) * q_w[i]);
    if (!write_kv) return;
    const int slot = slot_map[row];
    float sk = 0.f;
    for (int i = threadIdx.x; i < nk; i += blockDim.x) {
        const float v = to_f32(src[k_col + i]);
        sk = fmaf(v, v, sk);
    }
    sk = block_sum(sk, red);
    if (slot < 0) return;
    const float scale_k = 1.0f / sqrtf(sk / count_k + eps);
    const int page = slot / page_size, off = slot % page_size;
    for (int i = threadIdx.x; i < nk; i += blockDim.x) {
        const int g = i / hd, c = i - g * hd;
        T* kd = cache + ((((size_t)page * 2 + 0) * G + g) * page_size + off) * hd + c;
        T* vd = cache + ((((size_t)page * 2 + 1) * G + g) * page_size + off) * hd + c;
        *kd = from_f32<T>((to_f32(src[k_col + i]) * scale_k) * k_w[i]);
        *vd = src[v_col + i];
    }
}

extern "C" int kp_qk_rownorm_kv(const void* qkv, int ld, int k_col, int v_col, const float* q_w, const float* k_w, float eps,
                                float count_q, float count_k, const int* slot_map, void* q_out, int ldq, void* cache,
                                int page_size, int n, int H, int G, int hd, int write_kv, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (H < 1 || G < 1 || hd < 1 || !q_w || !q_out || (write_kv && (!k_w || !cache || !slot_map))) return KP_ERR_BAD_ARG;
    if (!(count_q > 0.f) || (write_kv && !(count_k > 0.f))) return KP_ERR_BAD_ARG;
    KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(qk_rownorm_kv_kernel<T>, dim3(n), dim3(256), 0, (cudaStream_t)stream, (const T*)qkv, ld,
                                               k_col, v_col, q_w, k_w, eps, count_q, count_k, slot_map, (T*)q_out, ldq, (T*)cache,
                                               page_size, H, G, hd, write_kv)));
    return kp_launch_status();
}

// ------------------------------------------------------------------------------------------------------------
// Means of blocks of `pool` positions: where a row of this step completes a block (its position p has (p + 1) % pool ==
// 0), the block's keys and values as the cache holds them are averaged (float32, summed in the order of the positions,
// whatever steps brought them there) and the means stored as entry p / pool of the request's pooled pages.
// pool_slot_map: the entry's slot a row, -1 for a row that completes no block.  VEC: elements a thread takes.
template <typename T, int VEC> struct PoolVec;
template <> struct PoolVec<bf16, 8> { typedef uint4 V; };
template <> struct PoolVec<float, 4> { typedef float4 V; };
template <> struct PoolVec<bf16, 1> { typedef bf16 V; };
template <> struct PoolVec<float, 1> { typedef float V; };

template <typename T, int VEC>
__global__ void __launch_bounds__(128)
pool_blocks_kernel(const T* __restrict__ cache, const int* __restrict__ block_table, int max_blocks, const int* __restrict__ row_seg,
                   const int* __restrict__ positions, const int* __restrict__ pool_slot_map, T* __restrict__ pool_cache, int pool,
                   int page_size, int planes_heads, int hd) {
    kp_pdl_begin();
    typedef typename PoolVec<T, VEC>::V V;
    const int row = blockIdx.y;
    const int slot = pool_slot_map[row];
    if (slot < 0) return;
    const int per = hd / VEC;
    const int i = blockIdx.x * blockDim.x + threadIdx.x;            // (K or V, head, stretch of the head)
    if (i >= planes_heads * per) return;
    const int head = i / per, c = (i - head * per) * VEC;
    const int p0 = positions[row] - pool + 1;
    const int* bt = block_table + (size_t)row_seg[row] * max_blocks;
    float acc[VEC];
#pragma unroll
    for (int j = 0; j < VEC; j++) acc[j] = 0.f;
#pragma unroll 4
    for (int k = 0; k < pool; k++) {
        const int pos = p0 + k;
        const V v = *reinterpret_cast<const V*>(cache + (((size_t)bt[pos / page_size] * planes_heads + head) * page_size + pos % page_size) * hd + c);
        const T* e = reinterpret_cast<const T*>(&v);
#pragma unroll
        for (int j = 0; j < VEC; j++) acc[j] += to_f32(e[j]);
    }
    V o;
    T* e = reinterpret_cast<T*>(&o);
#pragma unroll
    for (int j = 0; j < VEC; j++) e[j] = from_f32<T>(acc[j] / (float)pool);
    *reinterpret_cast<V*>(pool_cache + (((size_t)(slot / page_size) * planes_heads + head) * page_size + slot % page_size) * hd + c) = o;
}

extern "C" int kp_pool_blocks(const void* cache, const int* block_table, int max_blocks, const int* row_seg, const int* positions,
                              const int* pool_slot_map, void* pool_cache, int pool, int page_size, int n, int G, int hd, int dtype,
                              void* stream) {
    if (n <= 0) return 0;
    if (pool < 1 || page_size < 1 || G < 1 || hd < 1 || n > 65535) return KP_ERR_BAD_ARG;
    const int ph = 2 * G;
    cudaStream_t s = (cudaStream_t)stream;
#define POOL_LAUNCH(T, VEC)                                                                                               \
    kp_launch_pdl(pool_blocks_kernel<T, VEC>, dim3((ph * (hd / VEC) + 127) / 128, n), dim3(128), 0, s, (const T*)cache, block_table, \
                  max_blocks, row_seg, positions, pool_slot_map, (T*)pool_cache, pool, page_size, ph, hd)
    const bool aligned = !(((uintptr_t)cache | (uintptr_t)pool_cache) & 15);
    if (dtype == KP_DTYPE_BF16) {
        if (aligned && hd % 8 == 0) POOL_LAUNCH(bf16, 8); else POOL_LAUNCH(bf16, 1);
    } else if (dtype == KP_DTYPE_F32) {
        if (aligned && hd % 4 == 0) POOL_LAUNCH(float, 4); else POOL_LAUNCH(float, 1);
    } else {
        return KP_ERR_BAD_ARG;
    }
#undef POOL_LAUNCH
    return kp_launch_status();
}
