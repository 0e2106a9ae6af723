// Attention over a cache of latents: keys and values are expanded from one low-rank latent a token, k_h = Wuk_h c and
// v_h = Wuv_h c, beside a rotated key part that all heads share, and only the latent c and that part are kept.
//
//   cache row of a token: [ c (rank, normed; zeros up to rankp) | rotated key part (rot_dim; zeros up to rotp) | zeros up to W ]
//   s_h(t) = (q_h . Wuk_h c_t + qr_h . kr_t) scale ,  o_h = sum_t softmax(s_h)_t Wuv_h c_t        (causal)
//
// rankp and rotp are rank and rot_dim rounded up to 16, the row's W = rankp + rotp to 64; rows lie in pages
// [page][1][1][page_size][W].  Two ways of computing the same:
//
//  * absorbed (decoded tokens, short portions, the 32-bit mode): the expanding matrices move to the other side of the
//    sums, q'_h = Wuk_h^T q_h once a row, s_h(t) = ([q'_h | qr_h] . row_t) scale, u_h = sum_t softmax(s_h)_t c_t and
//    o_h = Wuv_h u_h.  All heads read the same rows, so a cache row is fetched once for up to 16 heads.  Per-head
//    products (head_gemm), a pass over chunks of keys (latent_split: bfloat16 on the tcgen05 tensor cores, or scalar) that
//    leaves each chunk's maximum, sum and unnormalised latent, and a merge in chunk order.
//  * expanded (prompt portions): the latents of the request's whole context are gathered from its pages, one product
//    expands them, and latent_prefill runs tiles of query rows over the expanded rows (128 rows on the tcgen05 tensor cores,
//    or 64 with mma.sync where the sizes are none of theirs).
//
// The softmax statistics are float32; its weights enter the products whole, as three bfloat16 parts.  The
// scalar form's chunks lie at multiples of 256 keys, so in the 32-bit mode the order of a row's sums does not depend on how its
// prompt was cut or on what else is in the batch; the tensor-core form makes its chunks as long as the step's rows allow
// (a few rows of short contexts still fill the device, and long ones are not cut finer than that needs), which
// moves the order of the float32 sums, nothing else.
#include "mma.cuh"
#include "tcgen05.cuh"

#define LA_CHUNK 256               // keys a chunk of the absorbed pass's scalar form
#define LA_SCALAR_HEADS 4          // heads a CTA of its scalar form
#define LP_TILE 64                 // query rows and keys a tile of the expanded form

KP_STATUS_WORD(g_latent_status, latent)          // 0 ok; 1: a bounded wait gave up

// Keys a chunk of the tensor-core form: so many tiles that n_chunks chunks reach the longest of the step's rows.  (Every
// CTA works it out from the rows' positions, one warp at a time; n_chunks is the host's choice.)
#define LT_TILE 64
__device__ __forceinline__ int lt_chunk_keys(const int* __restrict__ positions, int n_rows, int n_chunks) {
    int hi = 0;
    for (int i = threadIdx.x & 31; i < n_rows; i += 32) hi = max(hi, positions[i]);
    hi = __reduce_max_sync(0xffffffffu, hi);
    return (hi / LT_TILE + n_chunks) / n_chunks * LT_TILE;
}

// ------------------------------------------------------------------------------------------------ preparation
// One block a row of the input product p = [.. q: H heads of (dimp unrotated | rotp rotated) .. | latent (rankp) and key
// part (rotp) ..]: the latent normed over `rank` columns with weight w, and the key part rotated, go to the row's cache
// page; every head's rotated query part is rotated where it is, and for rows below n_absorbed also stored behind
// the place of the head's absorbed query in qa [n_absorbed][H][W].  rot: dimensions rotated (tables cos/sin
// [positions][rot / 2], which may carry a factor; null: no rotation).
template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_kernel(T* __restrict__ p, int ld, int q_col, int c_col, int H, int dimp, int rotp, int rank, int rankp,
                   int W, const float* __restrict__ w, float eps, const float* __restrict__ cos_tab, const float* __restrict__ sin_tab,
                   int rot, int interleaved, const int* __restrict__ positions, const int* __restrict__ slot_map,
                   T* __restrict__ cache, int page_size, T* __restrict__ qa, int n_absorbed) {
    kp_pdl_begin_early_if(gridDim.x > 1);
    __shared__ float red[32];
    const int row = blockIdx.x, tid = threadIdx.x;
    T* pr = p + (size_t)row * ld;
    const T* c = pr + c_col;
    const int pos = positions[row];
    const int half = cos_tab ? rot >> 1 : 0;
    const float* ct = cos_tab ? cos_tab + (size_t)pos * half : nullptr;
    const float* st = cos_tab ? sin_tab + (size_t)pos * half : nullptr;
    float ss = 0.f;
    for (int i = tid; i < rank; i += 256) { const float v = to_f32(c[i]); ss = fmaf(v, v, ss); }
    ss = block_sum(ss, red);
    const float scale = 1.0f / sqrtf(ss / (float)rank + eps);
    const int slot = cache ? slot_map[row] : -1;
    if (slot >= 0) {
        T* dst = cache + ((size_t)(slot / page_size) * page_size + slot % page_size) * W;
        for (int i = tid; i < rankp; i += 256) dst[i] = from_f32<T>(i < rank ? (to_f32(c[i]) * scale) * w[i] : 0.f);
        // (the key part's columns behind its own are zero in the product already)
        for (int i = tid; i < rotp; i += 256) {
            float v = to_f32(c[rankp + i]);
            if (i < 2 * half) {
                const int j = interleaved ? i >> 1 : (i < half ? i : i - half);
                const bool second = interleaved ? (i & 1) : i >= half;
                const float o = to_f32(c[rankp + (interleaved ? i ^ 1 : (second ? i - half : i + half))]);
                v = second ? o * st[j] + v * ct[j] : v * ct[j] - o * st[j];
            }
            dst[rankp + i] = from_f32<T>(v);
        }
        for (int i = rankp + rotp + tid; i < W; i += 256) dst[i] = from_f32<T>(0.f);
    }
    const int Dq = dimp + rotp;
    for (int i = tid; i < H * half; i += 256) {
        const int h = i / half, j = i - h * half;
        T* q = pr + q_col + (size_t)h * Dq + dimp;
        const int ia = interleaved ? 2 * j : j, ib = interleaved ? 2 * j + 1 : j + half;
        const float a = to_f32(q[ia]), b = to_f32(q[ib]);
        const T ra = from_f32<T>(a * ct[j] - b * st[j]), rb = from_f32<T>(a * st[j] + b * ct[j]);
        q[ia] = ra;
        q[ib] = rb;
        if (row < n_absorbed) {
            T* d = qa + ((size_t)row * H + h) * W + rankp;
            d[ia] = ra;
            d[ib] = rb;
        }
    }
    if (row < n_absorbed && W - rankp > 2 * half) {                // what is not rotated passes on as it is, and zeros behind
        const int rest = W - rankp - 2 * half;
        for (int i = tid; i < H * rest; i += 256) {
            const int h = i / rest, j = 2 * half + i % rest;
            qa[((size_t)row * H + h) * W + rankp + j] = j < rotp ? pr[q_col + (size_t)h * Dq + dimp + j] : from_f32<T>(0.f);
        }
    }
}

// The same for bfloat16 rows on 16-byte boundaries and interleaved pairs, four of them (eight elements) a thread: the row's
// query parts are fetched before the latent's sum is waited for.  Whole groups of four pairs are rotated (rot % 8 == 0, or
// nothing is).  PER: groups of eight query elements a thread at most.
template <int PER>
__global__ void __launch_bounds__(256)
latent_prep_vec_kernel(bf16* __restrict__ p, int ld, int q_col, int c_col, int H, int dimp, int rotp, int rank, int rankp, int W,
                       const float* __restrict__ w, float eps, const float* __restrict__ cos_tab, const float* __restrict__ sin_tab,
                       int rot, const int* __restrict__ positions, const int* __restrict__ slot_map, bf16* __restrict__ cache,
                       int page_size, bf16* __restrict__ qa, int n_absorbed) {
    kp_pdl_begin_early_if(gridDim.x > 1);
    __shared__ float red[32];
    const int row = blockIdx.x, tid = threadIdx.x;
    bf16* pr = p + (size_t)row * ld;
    const int pos = positions[row], half = rot >> 1;
    const float* ct = cos_tab ? cos_tab + (size_t)pos * half : nullptr;
    const float* st = cos_tab ? sin_tab + (size_t)pos * half : nullptr;
    const int Dq = dimp + rotp, gh = rotp >> 3, n_g = H * gh;      // groups a head, groups a row
    uint4 q[PER];
#pragma unroll
    for (int k = 0; k < PER; k++) {
        const int i = tid + k * 256;
        if (i < n_g) q[k] = *reinterpret_cast<const uint4*>(pr + q_col + (size_t)(i / gh) * Dq + dimp + (i % gh) * 8);
    }
    // the latent: rank / 8 groups and the key part behind it, one a thread (W <= 2048)
    const int ng = (rankp + rotp) >> 3;
    uint4 c = make_uint4(0, 0, 0, 0);
    float f[8];
    float ss = 0.f;
    if (tid < ng) c = *reinterpret_cast<const uint4*>(pr + c_col + tid * 8);
    {
        const __nv_bfloat162* c2 = reinterpret_cast<const __nv_bfloat162*>(&c);
#pragma unroll
        for (int j = 0; j < 4; j++) { const float2 x = __bfloat1622float2(c2[j]); f[2 * j] = x.x; f[2 * j + 1] = x.y; }
        if (tid * 8 < rankp) {                                     // (columns behind the rank are zero in the product)
#pragma unroll
            for (int j = 0; j < 8; j++) ss = fmaf(f[j], f[j], ss);
        }
    }
    ss = block_sum(ss, red);
    const float scale = 1.0f / sqrtf(ss / (float)rank + eps);
    auto rotate = [&](uint4 v, int g) {                            // group g of a rotated part
        if (ct == nullptr || g * 8 >= rot) return v;
        const float4 cc = __ldg(reinterpret_cast<const float4*>(ct + g * 4)), sn = __ldg(reinterpret_cast<const float4*>(st + g * 4));
        const float cs[4] = {cc.x, cc.y, cc.z, cc.w}, si[4] = {sn.x, sn.y, sn.z, sn.w};
        __nv_bfloat162* v2 = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const float2 x = __bfloat1622float2(v2[j]);
            v2[j] = __floats2bfloat162_rn(x.x * cs[j] - x.y * si[j], x.x * si[j] + x.y * cs[j]);
        }
        return v;
    };
    const int slot = cache ? slot_map[row] : -1;
    if (slot >= 0) {
        bf16* dst = cache + ((size_t)(slot / page_size) * page_size + slot % page_size) * W;
        if (tid * 8 < W) {
            uint4 o = make_uint4(0, 0, 0, 0);
            if (tid * 8 < rankp) {
                __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const int e = tid * 8 + 2 * j;
                    const float w0 = e < rank ? w[e] : 0.f, w1 = e + 1 < rank ? w[e + 1] : 0.f;
                    o2[j] = __floats2bfloat162_rn((f[2 * j] * scale) * w0, (f[2 * j + 1] * scale) * w1);
                }
            } else if (tid < ng) {
                o = rotate(c, tid - (rankp >> 3));
            }
            *reinterpret_cast<uint4*>(dst + tid * 8) = o;
        }
    }
#pragma unroll
    for (int k = 0; k < PER; k++) {
        const int i = tid + k * 256;
        if (i < n_g) {
            const int h = i / gh, g = i % gh;
            const uint4 v = rotate(q[k], g);
            if (ct != nullptr) *reinterpret_cast<uint4*>(pr + q_col + (size_t)h * Dq + dimp + g * 8) = v;
            if (row < n_absorbed) *reinterpret_cast<uint4*>(qa + ((size_t)row * H + h) * W + rankp + g * 8) = v;
        }
    }
    if (row < n_absorbed && W > rankp + rotp) {
        const int gz = (W - rankp - rotp) >> 3;
        for (int i = tid; i < H * gz; i += 256)
            *reinterpret_cast<uint4*>(qa + ((size_t)row * H + i / gz) * W + rankp + rotp + (i % gz) * 8) = make_uint4(0, 0, 0, 0);
    }
}

// ------------------------------------------------------------------------------------------- per-head products
// out[m, h, n] = sum_k a[m, h, k] b[h][n][k]   (times sigmoid(gate[m, h, n]) if gate).  Row and head strides are given.
// One CTA: 16 MT rows x 32 columns of one head, four warps of 8 columns; k in stretches of 64, double-buffered.
struct HeadGemmArgs {
    const void* a; const void* b; const void* gate; void* out;
    long long a_row, o_row, g_row;
    int a_head, o_head, g_head;
    int M, N, K, H;
};

template <int MT>
__global__ void __launch_bounds__(128)
head_gemm_mma_kernel(const HeadGemmArgs p) {
    constexpr int BK = 64, PITCH = BK + 8;
    kp_pdl_begin_early_if(p.M > 1);
    __shared__ __align__(16) bf16 As[2][MT * 16][PITCH], Bs[2][32][PITCH];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int n0 = blockIdx.x * 32, h = blockIdx.y, m0 = blockIdx.z * MT * 16;
    const bf16* A = (const bf16*)p.a + (size_t)h * p.a_head;
    const bf16* B = (const bf16*)p.b + (size_t)h * p.N * p.K;
    auto load = [&](int k0, int buf) {
        for (int i = tid; i < MT * 16 * 8; i += 128) {
            const int r = i >> 3, c = (i & 7) * 8;
            const bool ok = m0 + r < p.M && k0 + c < p.K;
            cp_async16(&As[buf][r][c], ok ? A + (size_t)(m0 + r) * p.a_row + k0 + c : A, ok);
        }
        for (int i = tid; i < 32 * 8; i += 128) {
            const int r = i >> 3, c = (i & 7) * 8;
            const bool ok = n0 + r < p.N && k0 + c < p.K;
            cp_async16(&Bs[buf][r][c], ok ? B + (size_t)(n0 + r) * p.K + k0 + c : B, ok);
        }
        cp_async_commit();
    };
    float acc[MT][4];
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int i = 0; i < 4; i++) acc[m][i] = 0.f;
    const int n_k = (p.K + BK - 1) / BK;
    load(0, 0);
    for (int it = 0; it < n_k; it++) {
        const int buf = it & 1;
        if (it + 1 < n_k) { load((it + 1) * BK, buf ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < BK / 16; ks += 2) {
            uint32_t b[4];                                         // 8 columns x 32 of k
            ldmatrix_x4(b, &Bs[buf][warp * 8 + (lane & 7)][ks * 16 + (lane >> 3) * 8]);
#pragma unroll
            for (int m = 0; m < MT; m++) {
                uint32_t a0[4], a1[4];
                ldmatrix_x4(a0, &As[buf][m * 16 + (lane & 15)][ks * 16 + (lane >> 4) * 8]);
                ldmatrix_x4(a1, &As[buf][m * 16 + (lane & 15)][ks * 16 + 16 + (lane >> 4) * 8]);
                mma_bf16(acc[m], a0[0], a0[1], a0[2], a0[3], b[0], b[1]);
                mma_bf16(acc[m], a1[0], a1[1], a1[2], a1[3], b[2], b[3]);
            }
        }
        __syncthreads();
    }
    const int n = n0 + warp * 8 + 2 * t;
    if (n >= p.N) return;                                          // (N is a multiple of 16: a pair is inside or outside)
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int half = 0; half < 2; half++) {
            const int r = m0 + m * 16 + g + half * 8;
            if (r >= p.M) continue;
            float v0 = acc[m][half * 2], v1 = acc[m][half * 2 + 1];
            if (p.gate) {
                const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>((const bf16*)p.gate + (size_t)r * p.g_row + (size_t)h * p.g_head + n));
                v0 /= 1.0f + expf(-z.x);
                v1 /= 1.0f + expf(-z.y);
            }
            *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)r * p.o_row + (size_t)h * p.o_head + n) = pack_bf16(v0, v1);
        }
}

// The same on the CUDA cores (float32 mode): 16 rows x 64 columns a CTA.
template <typename T>
__global__ void __launch_bounds__(256)
head_gemm_simt_kernel(const HeadGemmArgs p) {
    kp_pdl_begin();
    constexpr int BM = 16, BN = 64, BK = 16;
    __shared__ float As[BK][BM + 1], Bs[BK][BN + 1];
    const int tid = threadIdx.x, tx = tid & 63, ty = tid >> 6;     // column, row group of 4
    const int n0 = blockIdx.x * BN, h = blockIdx.y, m0 = blockIdx.z * BM;
    const T* A = (const T*)p.a + (size_t)h * p.a_head;
    const T* B = (const T*)p.b + (size_t)h * p.N * p.K;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < p.K; k0 += BK) {
        {
            const int r = tid >> 4, c = tid & 15;
            As[c][r] = (m0 + r < p.M && k0 + c < p.K) ? to_f32(A[(size_t)(m0 + r) * p.a_row + k0 + c]) : 0.f;
        }
        for (int i = tid; i < BN * BK; i += 256) {
            const int r = i >> 4, c = i & 15;
            Bs[c][r] = (n0 + r < p.N && k0 + c < p.K) ? to_f32(B[(size_t)(n0 + r) * p.K + k0 + c]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; k++)
#pragma unroll
            for (int i = 0; i < 4; i++) acc[i] = fmaf(As[k][ty * 4 + i], Bs[k][tx], acc[i]);
        __syncthreads();
    }
    const int n = n0 + tx;
    if (n >= p.N) return;
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int r = m0 + ty * 4 + i;
        if (r >= p.M) continue;
        float v = acc[i];
        if (p.gate) v /= 1.0f + expf(-to_f32(((const T*)p.gate)[(size_t)r * p.g_row + (size_t)h * p.g_head + n]));
        ((T*)p.out)[(size_t)r * p.o_row + (size_t)h * p.o_head + n] = from_f32<T>(v);
    }
}

// --------------------------------------------------------------------------------- absorbed pass, tensor cores
// One CTA: one chunk of one row's keys, NH (16 or 32) heads, on the 5th-generation tensor cores.  The keys stand where
// the tensor core wants many rows and the heads where it can do with few, so nothing is padded but the head count:
//
//   S^T = rows Q'^T    [keys x heads]: 64 cache rows a tile (K-major, as TMA brings them: boxes of 64 columns, 128-byte
//                      swizzle) times the absorbed queries, in MMAs of 64 x NH x 16.  Such an MMA leaves its rows in the lower
//                      half of every lane quarter; the odd boxes' sums go to the upper half, so that two chains run side
//                      by side and every lane has a part in what follows;
//   U^T = rows^T P^T   [latent columns x heads]: the same tile in shared memory, read as the MN-major operand in blocks of
//                      128 columns, times the softmax weights as 3 NH rows of bfloat16: the three parts of every
//                      head's float32 weights side by side, so that they enter whole for a few more columns.
//
// Roles by warp: 0 TMA (the queries once, a ring of tiles), 1 tensor memory and MMA of S, 2 - 9 two groups of four warps, a
// lane quarter each, 10 the MMA of U.  In the softmax of a tile a group has half of the heads, a lane 16 q + i of a quarter
// and its partner 16 lanes on the same key, half of those heads each; then all eight warps add U^T's columns (blocks shared
// among the groups) to their registers, rescaled by the heads' change of maximum, so that no pass over tensor memory
// rescales anything.  S and the weights are double-buffered: a tile's softmax runs while the tile before it is multiplied.
// Every wait is bounded; one that gives up sets the status word and an abort flag, and the CTA frees its tensor memory
// and returns.
#define LT_BOX_BYTES (LT_TILE * 128)                               // 64 rows x 64 columns of bfloat16
#define LT_MAX_STAGES 4
#define LT_THREADS 352

struct LatentSplitArgs {
    const int* block_table; const int* row_seg; const int* positions;
    float* part_acc; float* part_ml;
    int max_blocks, n_chunks, page_size, H, rankp, n_box, n_stages;
    float scale;
};

__device__ __forceinline__ float la_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int NH>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_split_tc_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmQ, const LatentSplitArgs p) {
    constexpr int HH = NH / 2, HQ = NH / 4;                        // heads a group has in the softmax, and a thread
    constexpr int NP = 3 * NH;                                     // columns of U^T in tensor memory, a block
    constexpr uint32_t TMEM_COLS = NH == 16 ? 256 : 512;           // S twice, four blocks of U^T
    extern __shared__ unsigned char lt_raw[];
    unsigned char* sm = lt_raw + ((1024u - (kp_smem_u32(lt_raw) & 1023u)) & 1023u);      // (by offset: it stays known as shared memory)
    const uint32_t tile_bytes = (uint32_t)p.n_box * LT_BOX_BYTES;
    unsigned char* Ks = sm;                                        // [n_stages][n_box][64 rows x 128 bytes]
    unsigned char* Qs = Ks + (size_t)p.n_stages * tile_bytes;      // [n_box][NH rows x 128 bytes]
    unsigned char* Ps = Qs + (size_t)p.n_box * NH * 128;           // [2][NP rows x 128 bytes]
    float* max_s = reinterpret_cast<float*>(Ps + 2 * NP * 128);    // [2 tiles][NH][4 quarters]
    float* sum_s = max_s + 8 * NH;                                 // [NH][4 quarters]
    float* corr_s = sum_s + 4 * NH;                                // [4 tiles][NH]
    uint64_t* bars = reinterpret_cast<uint64_t*>(corr_s + 4 * NH);
    uint64_t* q_full = bars;
    uint64_t* k_full = bars + 1;                                   // [LT_MAX_STAGES]
    uint64_t* k_empty = k_full + LT_MAX_STAGES;                    // [LT_MAX_STAGES]
    uint64_t* s_full = k_empty + LT_MAX_STAGES;                    // [2]
    uint64_t* p_full = s_full + 2;                                 // [2]
    uint64_t* u_full = p_full + 2;
    uint64_t* u_empty = u_full + 1;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(u_empty + 1);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        kp_mbar_init(q_full, 1);
        for (int s = 0; s < LT_MAX_STAGES; s++) { kp_mbar_init(&k_full[s], 1); kp_mbar_init(&k_empty[s], 1); }
        for (int b = 0; b < 2; b++) { kp_mbar_init(&s_full[b], 1); kp_mbar_init(&p_full[b], 256); }
        kp_mbar_init(u_full, 1);
        kp_mbar_init(u_empty, 8);
        *abort_flag = 0;
        kp_mbar_init_fence();
    }
    kp_pdl_begin_early_if(gridDim.z > 1);
    // (the whole CTA leaves here or stays: tensor memory is taken only by one that stays)
    const int chunk = blockIdx.x, h0 = blockIdx.y * NH, row = blockIdx.z;
    const int k_hi = p.positions[row], seg = p.row_seg[row], ck = lt_chunk_keys(p.positions, gridDim.z, p.n_chunks), c0 = chunk * ck;
    if (c0 > k_hi) return;
    const int n_keys = min(k_hi + 1 - c0, ck), n_tiles = (n_keys + LT_TILE - 1) / LT_TILE;
    if (warp == 1) kp_tmem_alloc(tmem_slot, TMEM_COLS);
    kp_tc_fence_before();
    __syncthreads();
    kp_tc_fence_after();
    const uint32_t tmem_s = *tmem_slot, tmem_u = tmem_s + 2 * NH;
    const int n_blk = (p.rankp + 127) / 128;

    if (warp == 0) {
        if (lane == 0) {
            const int* bt = p.block_table + (size_t)seg * p.max_blocks;
            const int box = min(p.page_size, LT_TILE);             // rows a load
            for (int it = 0; it < n_tiles; it++) {
                const int s = it % p.n_stages;
                if (*abort_flag || !kp_mbar_wait_bounded(&k_empty[s], ((it / p.n_stages) & 1) ^ 1)) { *abort_flag = 1; break; }
                const int t0 = it * LT_TILE;                       // first key of the tile, counted from the chunk's
                const int n_boxes = (min(LT_TILE, n_keys - t0) + box - 1) / box;
                kp_mbar_expect_tx(&k_full[s], (uint32_t)(n_boxes * box * 128 * p.n_box));
                for (int b = 0; b < n_boxes; b++) {
                    const int key = c0 + t0 + b * box;
                    const int y = bt[key / p.page_size] * p.page_size + key % p.page_size;
                    unsigned char* dst = Ks + (size_t)s * tile_bytes + (size_t)b * box * 128;
                    if (box == LT_TILE) kp_tma_load_3d(dst, &tmC, 0, y, 0, &k_full[s]);      // the whole tile
                    else                                           // (smaller pages: a load a group of columns, which lie a tile apart)
                        for (int j = 0; j < p.n_box; j++) kp_tma_load_3d(dst + (size_t)j * LT_BOX_BYTES, &tmC, 0, y, j, &k_full[s]);
                }
                if (it == 0) {                                     // (behind the first tile, which takes longer to come)
                    kp_mbar_expect_tx(q_full, (uint32_t)p.n_box * NH * 128);
                    kp_tma_load_3d(Qs, &tmQ, 0, row * p.H + h0, 0, q_full);
                }
            }
        }
    } else if (warp == 1) {
        // ---- S^T of tile it: the tile has come, and the softmax has read what stood in its columns (all lanes in step, an
        // elected one issues)
        constexpr uint32_t idesc_s = kp_umma_idesc(64, NH);
        const uint64_t k_desc = kp_umma_desc(kp_smem_u32(Ks)), q_desc = kp_umma_desc(kp_smem_u32(Qs));
        bool ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(q_full, 0));
        for (int it = 0; it < n_tiles && ok; it++) {
            const int s = it % p.n_stages;
            ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(&k_full[s], (it / p.n_stages) & 1));
            if (ok && it > 1) ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(&p_full[it & 1], ((it - 2) >> 1) & 1));
            if (!ok || __any_sync(0xffffffffu, *abort_flag)) { ok = false; break; }
            kp_tc_fence_after();
            const uint64_t kd = k_desc + s * (tile_bytes >> 4);    // (the address is the descriptor's low field, in 16 bytes)
            const uint32_t d = tmem_s + (it & 1) * NH;
            for (int j = 0; j < p.n_box; j++)
                kp_umma_bf16_box(d + ((uint32_t)(j & 1) << 20), kd + j * (LT_BOX_BYTES >> 4), q_desc + j * (NH * 128 >> 4), idesc_s, j > 1);
            kp_umma_commit_warp(&s_full[it & 1]);
        }
        if (!ok) *abort_flag = 1;
    } else if (warp == 10) {
        // ---- U^T of tile it: its weights are there, and U of the tile before has been read
        constexpr uint32_t idesc_u = kp_umma_idesc(128, NP, false, true);
        const uint64_t v_desc = kp_umma_desc_mn(kp_smem_u32(Ks), LT_BOX_BYTES), p_desc = kp_umma_desc(kp_smem_u32(Ps));
        bool ok = true;
        for (int it = 0; it < n_tiles && ok; it++) {
            const int s = it % p.n_stages;
            ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(&p_full[it & 1], (it >> 1) & 1));
            if (ok && it > 0) ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(u_empty, (it - 1) & 1));
            if (!ok || __any_sync(0xffffffffu, *abort_flag)) { ok = false; break; }
            kp_tc_fence_after();
            const uint64_t vd = v_desc + s * (tile_bytes >> 4), pd = p_desc + (it & 1) * (NP * 128 >> 4);
            for (int m = 0; m < n_blk; m++) {
#pragma unroll
                for (int kk = 0; kk < LT_TILE / 16; kk++)
                    kp_umma_bf16_warp(tmem_u + m * NP, vd + m * (2 * LT_BOX_BYTES >> 4) + kk * (2048 >> 4), pd + 2 * kk, idesc_u, kk ? 1u : 0u);
            }
            kp_umma_commit_warp(u_full);
            kp_umma_commit_warp(&k_empty[s]);
        }
        if (!ok) *abort_flag = 1;
    } else {
        const int grp = (warp - 2) >> 2, q4 = warp & 3;            // (a warp reads lanes 32 (warp % 4) .. of tensor memory)
        const uint32_t lane_off = (uint32_t)(q4 * 32) << 16;
        const bool upper = lane >= 16;
        const int key = q4 * 16 + (lane & 15);                     // of the tile
        const int head0 = grp * HH + (upper ? HQ : 0);             // this thread's heads in the softmax: HQ from here on
        const float sl2 = p.scale * 1.4426950408889634f;           // scores in units of log2
        float m_run[HQ], l_run[HQ];
#pragma unroll
        for (int h = 0; h < HQ; h++) { m_run[h] = -INFINITY; l_run[h] = 0.f; }
        float acc[2][NH];
#pragma unroll
        for (int b = 0; b < 2; b++)
#pragma unroll
            for (int h = 0; h < NH; h++) acc[b][h] = 0.f;
        bool ok = true;
        // The warps of a group meet at a barrier in every tile, so they go on or leave together: a wait that gave up is
        // only noted (`ok`), and the barrier tells all (its result: do all say ok?).
        auto agree = [&](bool mine) {
            uint32_t r;
            asm volatile("{\n .reg .pred a, b;\n setp.ne.u32 a, %1, 0;\n barrier.cta.red.and.pred b, %2, 128, a;\n selp.u32 %0, 1, 0, b;\n}"
                         : "=r"(r) : "r"(mine ? 1u : 0u), "r"(1 + grp) : "memory");
            return r != 0;
        };
        auto softmax = [&](int it) {                               // false: the warps of the group leave
            const int b = it & 1, s = it % p.n_stages;
            if (ok && (!kp_mbar_wait_bounded(&s_full[b], (it >> 1) & 1) || *abort_flag)) ok = false;
            kp_tc_fence_after();
            const int valid = min(LT_TILE, n_keys - it * LT_TILE);
            float v[HQ];
            {
                uint32_t raw[HH];
                if constexpr (HH == 8) kp_tmem_ld8_issue(tmem_s + b * NH + grp * HH + lane_off, raw);
                else kp_tmem_ld16_issue(tmem_s + b * NH + grp * HH + lane_off, raw);
                kp_tmem_ld_wait();
                // the even boxes' sums are in the lower lanes, the odd boxes' in the upper ones (if there are any)
#pragma unroll
                for (int h = 0; h < HQ; h++) {
                    const float lo = __uint_as_float(raw[h]), hi = __uint_as_float(raw[HQ + h]);
                    const float other = __shfl_xor_sync(0xffffffffu, upper ? lo : hi, 16);
                    const float sum = p.n_box > 1 ? (upper ? hi : lo) + other : (upper ? other : lo);
                    v[h] = key < valid ? sum * sl2 : -INFINITY;
                }
            }
            if (valid < LT_TILE) {
                // the chunk's last tile: rows that no copy of this tile filled, or that hold another request's keys, meet
                // weights of 0 below and are cleared (0 times NaN is not 0); S has read them already
                unsigned char* kt = Ks + (size_t)s * tile_bytes;
                const int n = (LT_TILE - valid) * 2 * n_blk;       // (row, box) pairs
                const int n_real = min(2 * n_blk, p.n_box);
                for (int i = threadIdx.x - 64; i < n; i += 256) {
                    const int r = valid + i / (2 * n_blk), j = i % (2 * n_blk);
                    if (j >= n_real) continue;
                    uint4* d = reinterpret_cast<uint4*>(kt + (size_t)j * LT_BOX_BYTES + r * 128);
#pragma unroll
                    for (int c = 0; c < 8; c++) d[c] = make_uint4(0, 0, 0, 0);
                }
            }
            // the tile's maximum of every head: over the half warp's keys, then over the four warps of the group
            float* mx = max_s + b * 4 * NH;
            float mine = 0.f;
#pragma unroll
            for (int h = 0; h < HQ; h++) {
                float w = v[h];
#pragma unroll
                for (int o = 8; o > 0; o >>= 1) w = fmaxf(w, __shfl_xor_sync(0xffffffffu, w, o));
                if ((lane & 15) == h) mine = w;
            }
            if ((lane & 15) < HQ) mx[(head0 + (lane & 15)) * 4 + q4] = mine;
            if (!agree(ok)) { ok = false; return false; }
            unsigned char* pr = Ps + (size_t)b * (NP * 128) + (key & 7) * 2;
#pragma unroll
            for (int h = 0; h < HQ; h++) {
                const int hh = head0 + h;
                const float4 m4 = *reinterpret_cast<const float4*>(mx + hh * 4);
                const float m_new = fmaxf(fmaxf(m_run[h], fmaxf(m4.x, m4.y)), fmaxf(m4.z, m4.w));   // (finite: a tile's first key is the row's)
                const float corr = la_exp2(m_run[h] - m_new);      // (2^-inf = 0 for the first tile)
                float w = la_exp2(v[h] - m_new);
                m_run[h] = m_new;
                l_run[h] = fmaf(l_run[h], corr, w);
                if (key == 0) corr_s[(it & 3) * NH + hh] = corr;
#pragma unroll
                for (int part = 0; part < 3; part++) {
                    const bf16 x = __float2bfloat16_rn(w);
                    w -= __bfloat162float(x);
                    const int n = part * NH + hh;
                    *reinterpret_cast<bf16*>(pr + n * 128 + (((key >> 3) ^ (n & 7)) << 4)) = x;
                }
            }
            kp_tc_fence_before();                                  // the reads of S are done
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // the weights and cleared rows are read by the tensor core
            kp_mbar_arrive(&p_full[b]);
            return true;
        };
        auto gather = [&](int it) {
            if (!kp_mbar_wait_bounded(u_full, it & 1) || *abort_flag) { ok = false; return; }
            kp_tc_fence_after();
            const float* corr = corr_s + (it & 3) * NH;
#pragma unroll
            for (int b = 0; b < 2; b++) {
                const int m = grp + 2 * b;                         // the group's blocks of 128 columns
                if (m < n_blk) {
                    const uint32_t ta = tmem_u + m * NP + lane_off;
                    if constexpr (NH == 16) {
                        uint32_t u[3][16];
#pragma unroll
                        for (int part = 0; part < 3; part++) kp_tmem_ld16_issue(ta + part * NH, u[part]);
                        kp_tmem_ld_wait();
#pragma unroll
                        for (int h = 0; h < 16; h++)
                            acc[b][h] = fmaf(acc[b][h], corr[h], __uint_as_float(u[0][h]) + (__uint_as_float(u[1][h]) + __uint_as_float(u[2][h])));
                    } else {
#pragma unroll
                        for (int half = 0; half < 2; half++) {
                            uint32_t u[3][16];
#pragma unroll
                            for (int part = 0; part < 3; part++) kp_tmem_ld16_issue(ta + part * NH + half * 16, u[part]);
                            kp_tmem_ld_wait();
#pragma unroll
                            for (int h = 0; h < 16; h++)
                                acc[b][half * 16 + h] = fmaf(acc[b][half * 16 + h], corr[half * 16 + h],
                                                             __uint_as_float(u[0][h]) + (__uint_as_float(u[1][h]) + __uint_as_float(u[2][h])));
                        }
                    }
                }
            }
            kp_tc_fence_before();
            __syncwarp();
            if (lane == 0) kp_mbar_arrive(u_empty);
        };
        bool together = softmax(0);
        for (int it = 0; it < n_tiles && together; it++) {
            if (it + 1 < n_tiles) together = softmax(it + 1);
            if (ok) gather(it);
        }
        if (together) {
            // the tiles' sums of weights: over the half warp, then over the four warps of the group
#pragma unroll
            for (int h = 0; h < HQ; h++) {
                float l = l_run[h];
#pragma unroll
                for (int o = 8; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
                if ((lane & 15) == 0) sum_s[(head0 + h) * 4 + q4] = l;
            }
            ok = agree(ok);
        }
        if (!ok) *abort_flag = 1;
        if (ok) {
            const int nh = min(NH, p.H - h0);
#pragma unroll
            for (int b = 0; b < 2; b++) {
                const int col = (grp + 2 * b) * 128 + q4 * 32 + lane;
                if (col < p.rankp) {
#pragma unroll
                    for (int h = 0; h < NH; h++)
                        if (h < nh) p.part_acc[(((size_t)row * p.H + h0 + h) * p.n_chunks + chunk) * p.rankp + col] = acc[b][h];
                }
            }
            if (key == 0) {
#pragma unroll
                for (int h = 0; h < HQ; h++) {
                    const int hh = head0 + h;
                    const float4 l4 = *reinterpret_cast<const float4*>(sum_s + hh * 4);
                    if (hh < nh)
                        *reinterpret_cast<float2*>(p.part_ml + (((size_t)row * p.H + h0 + hh) * p.n_chunks + chunk) * 2) =
                            make_float2(m_run[h] * 0.6931471805599453f, (l4.x + l4.y) + (l4.z + l4.w));
                }
            }
        }
    }
    kp_tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        if (threadIdx.x == 0) atomicExch(&g_latent_status, 1);
        kp_linger_after_failure();
    }
    if (warp == 1) kp_tmem_dealloc(tmem_s, TMEM_COLS);
}

// ------------------------------------------------------------------------------------- absorbed pass, CUDA cores
// The same for any sizes and both storage types: one CTA a (chunk, up to 4 heads, row); a key a thread for the scores,
// a column a thread for the sums.
template <typename T>
__global__ void __launch_bounds__(LA_CHUNK)
latent_split_kernel(const T* __restrict__ qa, const T* __restrict__ cache, const int* __restrict__ block_table, int max_blocks,
                    const int* __restrict__ row_seg, const int* __restrict__ positions, float* __restrict__ part_acc,
                    float* __restrict__ part_ml, int n_chunks, float scale, int page_size, int H, int rankp, int W) {
    kp_pdl_begin();
    constexpr int R = LA_SCALAR_HEADS;
    extern __shared__ __align__(16) float ls_smem[];               // [R][W] queries, [R][256] weights, [32], [256] row offsets
    float* qs = ls_smem;
    float* ps = qs + R * W;
    float* red = ps + R * LA_CHUNK;
    int* where = reinterpret_cast<int*>(red + 32);
    const int tid = threadIdx.x, chunk = blockIdx.x, h0 = blockIdx.y * R, row = blockIdx.z;
    const int k_hi = positions[row], c0 = chunk * LA_CHUNK;
    if (c0 > k_hi) return;
    const int n_keys = min(k_hi + 1 - c0, LA_CHUNK), nh = min(R, H - h0);
    const int* bt = block_table + (size_t)row_seg[row] * max_blocks;
    for (int i = tid; i < R * W; i += LA_CHUNK) qs[i] = i < nh * W ? to_f32(qa[((size_t)row * H + h0) * W + i]) : 0.f;
    const int key = c0 + tid;
    where[tid] = tid < n_keys ? bt[key / page_size] * page_size + key % page_size : 0;
    __syncthreads();
    float s[R];
#pragma unroll
    for (int r = 0; r < R; r++) s[r] = 0.f;
    if (tid < n_keys) {
        const T* kp = cache + (size_t)where[tid] * W;
        constexpr int VN = 16 / sizeof(T);
        for (int i = 0; i < W; i += VN) {                          // (W is a multiple of 16)
            const uint4 raw = *reinterpret_cast<const uint4*>(kp + i);
            const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
            for (int j = 0; j < VN; j++) {
                const float kv = to_f32(e[j]);
#pragma unroll
                for (int r = 0; r < R; r++) s[r] = fmaf(qs[r * W + i + j], kv, s[r]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; r++) {
        const float v = tid < n_keys ? s[r] * scale : -INFINITY;
        const float m = block_max(v, red);
        const float p = tid < n_keys ? expf(v - m) : 0.f;
        const float l = block_sum(p, red);
        ps[r * LA_CHUNK + tid] = p;
        if (tid == 0 && r < nh) {
            float* ml = part_ml + (((size_t)row * H + h0 + r) * n_chunks + chunk) * 2;
            ml[0] = m;
            ml[1] = l;
        }
    }
    __syncthreads();
    for (int c = tid; c < rankp; c += LA_CHUNK) {
        float acc[R];
#pragma unroll
        for (int r = 0; r < R; r++) acc[r] = 0.f;
#pragma unroll 4
        for (int k = 0; k < n_keys; k++) {
            const float v = to_f32(cache[(size_t)where[k] * W + c]);
#pragma unroll
            for (int r = 0; r < R; r++) acc[r] = fmaf(ps[r * LA_CHUNK + k], v, acc[r]);
        }
#pragma unroll
        for (int r = 0; r < R; r++)
            if (r < nh) part_acc[(((size_t)row * H + h0 + r) * n_chunks + chunk) * rankp + c] = acc[r];
    }
}

// The chunks of a (head, row) put together in chunk order: u = sum_c acc_c exp(m_c - m) / sum_c l_c exp(m_c - m).
template <typename T>
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml, const int* __restrict__ positions,
                    T* __restrict__ out, int n_chunks, int H, int rankp, int fixed_chunk) {
    kp_pdl_begin_early_if(gridDim.y > 1);
    extern __shared__ float lm_w[];                                // [n_chunks] weights, [32]
    float* red = lm_w + n_chunks;
    const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
    const int pos = positions[row];
    const int n = min(pos / (fixed_chunk ? LA_CHUNK : lt_chunk_keys(positions, gridDim.y, n_chunks)) + 1, n_chunks);
    const float* ml = part_ml + ((size_t)row * H + h) * n_chunks * 2;
    float m = -INFINITY;
    for (int c = tid; c < n; c += 128) { const float v = ml[2 * c]; lm_w[c] = v; m = fmaxf(m, v); }
    m = block_max(m, red);
    for (int c = tid; c < n; c += 128) lm_w[c] = expf(lm_w[c] - m);
    __syncthreads();
    float l = 0.f;
    for (int c = 0; c < n; c++) l = fmaf(ml[2 * c + 1], lm_w[c], l);
    const float inv = 1.0f / l;
    const float* pa = part_acc + ((size_t)row * H + h) * n_chunks * rankp;
    for (int i = tid * 4; i < rankp; i += 512) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int c = 0; c < n; c++) {
            const float4 a = *reinterpret_cast<const float4*>(pa + (size_t)c * rankp + i);
            const float w = lm_w[c];
            v.x = fmaf(a.x, w, v.x); v.y = fmaf(a.y, w, v.y); v.z = fmaf(a.z, w, v.z); v.w = fmaf(a.w, w, v.w);
        }
        T* o = out + ((size_t)row * H + h) * rankp + i;
        o[0] = from_f32<T>(v.x * inv); o[1] = from_f32<T>(v.y * inv); o[2] = from_f32<T>(v.z * inv); o[3] = from_f32<T>(v.w * inv);
    }
}

// ---------------------------------------------------------------------------------------------- expanded pass
// The cache rows of the contexts of some segments, side by side: row ctx_base[i] + t of `out` [T][W] is key t of segment i
// (segments without rows there have ctx_base[i] == ctx_base[i + 1]).  A warp a row.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const bf16* __restrict__ cache, const int* __restrict__ block_table, int max_blocks, const int* __restrict__ ctx_base,
                     int n_seg, bf16* __restrict__ out, int n_rows, int page_size, int W) {
    kp_pdl_begin();
    const int lane = threadIdx.x & 31, r = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (r >= n_rows) return;
    int lo = 0, hi = n_seg;                                        // the last segment with ctx_base <= r
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (ctx_base[mid] <= r) lo = mid; else hi = mid;
    }
    const int key = r - ctx_base[lo];
    const uint4* src = reinterpret_cast<const uint4*>(cache + ((size_t)block_table[(size_t)lo * max_blocks + key / page_size] * page_size + key % page_size) * W);
    uint4* dst = reinterpret_cast<uint4*>(out + (size_t)r * W);
    for (int i = lane; i < W >> 3; i += 32) dst[i] = src[i];
}

// One CTA: 64 query rows of a segment, one head: 4 warps x 16 rows over tiles of 64 keys, double-buffered (cp.async).  A
// tile's key rows are [expanded unrotated part | shared rotated part], its value rows the expanded values.  KS, VT: the most
// 16-column steps of a key and 8-column tiles of a value.
struct LatentPrefillArgs {
    const bf16* q; const bf16* ex; const bf16* rows; bf16* out;
    const int* cu_rows; const int* seg_pos; const int* tile_seg; const int* tile_row0; const int* ctx_base;
    int ldq, ldo, ld_ex, W, rankp, dimp, rotp, vdimp, v_col, n_tiles;
    float scale;
};

template <int KS, int VT>
__global__ void __launch_bounds__(128)
latent_prefill_kernel(const LatentPrefillArgs p) {
    kp_pdl_begin();
    extern __shared__ __align__(128) unsigned char lp_smem[];
    const int Dq = p.dimp + p.rotp, kp = Dq + 8, vp = p.vdimp + 8;
    bf16* Ks = reinterpret_cast<bf16*>(lp_smem);                   // [2][64][kp]
    bf16* Vs = Ks + (size_t)2 * LP_TILE * kp;                      // [2][64][vp]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, tile = p.n_tiles - 1 - blockIdx.x;   // (later rows of a prompt read more keys: they go first)
    const int seg = p.tile_seg[tile], row0 = p.tile_row0[tile];
    const int n_rows = min(LP_TILE, p.cu_rows[seg + 1] - row0);
    const int pos0 = p.seg_pos[seg] + (row0 - p.cu_rows[seg]);
    const int k_hi = pos0 + n_rows - 1, n_kt = k_hi / LP_TILE + 1;
    const size_t base = p.ctx_base[seg];
    const int nks = Dq >> 4, nvt = p.vdimp >> 3;
    const int kc = p.dimp >> 3, rc = p.rotp >> 3, vc = p.vdimp >> 3;       // 16-byte pieces

    auto load = [&](int kt, int buf) {
        bf16* kd = Ks + (size_t)buf * LP_TILE * kp;
        bf16* vd = Vs + (size_t)buf * LP_TILE * vp;
        const int per = kc + rc + vc;
        for (int i = tid; i < LP_TILE * per; i += 128) {
            const int r = i / per, c = i - r * per, key = kt * LP_TILE + r;
            const bool ok = key <= k_hi;
            const size_t er = base + (ok ? key : 0);
            const bf16* src;
            bf16* dst;
            if (c < kc) { src = p.ex + er * p.ld_ex + (size_t)h * p.dimp + c * 8; dst = kd + (size_t)r * kp + c * 8; }
            else if (c < kc + rc) { src = p.rows + er * p.W + p.rankp + (c - kc) * 8; dst = kd + (size_t)r * kp + c * 8; }
            else { src = p.ex + er * p.ld_ex + p.v_col + (size_t)h * p.vdimp + (c - kc - rc) * 8; dst = vd + (size_t)r * vp + (c - kc - rc) * 8; }
            cp_async16(dst, src, ok);
        }
        cp_async_commit();
    };
    load(0, 0);

    const int ra = warp * 16 + g, rb = ra + 8;
    const int pos_a = pos0 + ra, pos_b = pos0 + rb;
    const bool has_a = ra < n_rows, has_b = rb < n_rows;
    uint32_t qf[KS][4];
    {
        const bf16* qa = p.q + (size_t)(row0 + min(ra, n_rows - 1)) * p.ldq + (size_t)h * Dq;
        const bf16* qb = p.q + (size_t)(row0 + min(rb, n_rows - 1)) * p.ldq + (size_t)h * Dq;
#pragma unroll
        for (int ks = 0; ks < KS; ks++) {
            if (ks < nks) {
                qf[ks][0] = *reinterpret_cast<const uint32_t*>(qa + ks * 16 + 2 * t);
                qf[ks][1] = *reinterpret_cast<const uint32_t*>(qb + ks * 16 + 2 * t);
                qf[ks][2] = *reinterpret_cast<const uint32_t*>(qa + ks * 16 + 8 + 2 * t);
                qf[ks][3] = *reinterpret_cast<const uint32_t*>(qb + ks * 16 + 8 + 2 * t);
            }
        }
    }
    float o[VT][4];
#pragma unroll
    for (int d = 0; d < VT; d++)
#pragma unroll
        for (int i = 0; i < 4; i++) o[d][i] = 0.f;
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;

    for (int kt = 0; kt < n_kt; kt++) {
        const int buf = kt & 1;
        if (kt + 1 < n_kt) { load(kt + 1, buf ^ 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const int t0 = kt * LP_TILE;
        const int w_hi = pos0 + min(warp * 16 + 15, n_rows - 1);
        if (warp * 16 < n_rows && t0 <= w_hi) {
            const bf16* Kt = Ks + (size_t)buf * LP_TILE * kp;
            const bf16* Vt = Vs + (size_t)buf * LP_TILE * vp;
            float s[8][4];
#pragma unroll
            for (int nt = 0; nt < 8; nt++)
#pragma unroll
                for (int i = 0; i < 4; i++) s[nt][i] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KS; ks++) {
                if (ks < nks) {
#pragma unroll
                    for (int nt = 0; nt < 8; nt += 2) {
                        uint32_t b[4];
                        ldmatrix_x4(b, Kt + (size_t)((nt + (lane >> 4)) * 8 + (lane & 7)) * kp + ks * 16 + ((lane >> 3) & 1) * 8);
                        mma_bf16(s[nt], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b[0], b[1]);
                        mma_bf16(s[nt + 1], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b[2], b[3]);
                    }
                }
            }
            float mx_a = -INFINITY, mx_b = -INFINITY;
#pragma unroll
            for (int nt = 0; nt < 8; nt++) {
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    const int key = t0 + nt * 8 + 2 * t + i;
                    s[nt][i] = has_a && key <= pos_a ? s[nt][i] * p.scale : -INFINITY;
                    s[nt][2 + i] = has_b && key <= pos_b ? s[nt][2 + i] * p.scale : -INFINITY;
                    mx_a = fmaxf(mx_a, s[nt][i]);
                    mx_b = fmaxf(mx_b, s[nt][2 + i]);
                }
            }
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1));
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
            mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1));
            mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
            const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
            const float ca = m_a == -INFINITY ? 0.f : expf(m_a - mn_a), cb = m_b == -INFINITY ? 0.f : expf(m_b - mn_b);
            float sa = 0.f, sb = 0.f;
#pragma unroll
            for (int nt = 0; nt < 8; nt++) {
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    s[nt][i] = mn_a == -INFINITY ? 0.f : expf(s[nt][i] - mn_a);
                    s[nt][2 + i] = mn_b == -INFINITY ? 0.f : expf(s[nt][2 + i] - mn_b);
                    sa += s[nt][i];
                    sb += s[nt][2 + i];
                }
            }
            sa += __shfl_xor_sync(0xffffffffu, sa, 1); sa += __shfl_xor_sync(0xffffffffu, sa, 2);
            sb += __shfl_xor_sync(0xffffffffu, sb, 1); sb += __shfl_xor_sync(0xffffffffu, sb, 2);
            l_a = l_a * ca + sa; l_b = l_b * cb + sb;
            m_a = mn_a; m_b = mn_b;
#pragma unroll
            for (int d = 0; d < VT; d++) { o[d][0] *= ca; o[d][1] *= ca; o[d][2] *= cb; o[d][3] *= cb; }
#pragma unroll
            for (int kk = 0; kk < 4; kk++) {                       // 16 keys at a time: their weights' three parts, then V once
                uint32_t pf[3][4];
#pragma unroll
                for (int part = 0; part < 3; part++) {
                    pf[part][0] = pack_bf16_part(s[2 * kk][0], s[2 * kk][1]);
                    pf[part][1] = pack_bf16_part(s[2 * kk][2], s[2 * kk][3]);
                    pf[part][2] = pack_bf16_part(s[2 * kk + 1][0], s[2 * kk + 1][1]);
                    pf[part][3] = pack_bf16_part(s[2 * kk + 1][2], s[2 * kk + 1][3]);
                }
#pragma unroll
                for (int d = 0; d < VT; d += 2) {
                    if (d < nvt) {
                        uint32_t b[4];
                        ldmatrix_x4_trans(b, Vt + (size_t)(kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * vp + (d + (lane >> 4)) * 8);
#pragma unroll
                        for (int part = 0; part < 3; part++) {
                            mma_bf16(o[d], pf[part][0], pf[part][1], pf[part][2], pf[part][3], b[0], b[1]);
                            mma_bf16(o[d + 1], pf[part][0], pf[part][1], pf[part][2], pf[part][3], b[2], b[3]);
                        }
                    }
                }
            }
        }
        __syncthreads();                                           // the buffer is free for the load after next
    }
    const float ia = l_a > 0.f ? 1.0f / l_a : 0.f, ib = l_b > 0.f ? 1.0f / l_b : 0.f;
#pragma unroll
    for (int d = 0; d < VT; d++) {
        if (d >= nvt) continue;
        const size_t col = (size_t)h * p.vdimp + d * 8 + 2 * t;
        if (has_a) *reinterpret_cast<uint32_t*>(p.out + (size_t)(row0 + ra) * p.ldo + col) = pack_bf16(o[d][0] * ia, o[d][1] * ia);
        if (has_b) *reinterpret_cast<uint32_t*>(p.out + (size_t)(row0 + rb) * p.ldo + col) = pack_bf16(o[d][2] * ib, o[d][3] * ib);
    }
}

// The expanded pass on the 5th-generation tensor cores: one CTA takes 128 query rows of a segment and one head, over tiles of
// 64 keys.
//
//   S  = Q K^T     128 x 64: Q and the tile's key parts K-major, by TMA (boxes of 64 columns, 128-byte swizzle): the expanded
//                  unrotated part and the shared rotated part stand in boxes of their own, and only the steps of 16
//                  columns that the parts have are multiplied;
//   PV = P V       128 x vdimp: the float32 weights as three bfloat16 parts, multiplied one after the other into the same
//                  columns, so that they enter whole; V as it lies (keys x columns: the MN-major operand).
//
// Roles by warp: 0 TMA (Q once, a ring of two tiles), 1 tensor memory and MMA of S, 2 - 9 the rows, 10 MMA of PV.  A row has
// two threads (two groups of four warps, a lane quarter each): both take the maximum of its 64 scores, each the exponentials
// of half of its keys and the sums of half of its value columns, which stay in registers and are rescaled there, so
// nothing rescales tensor memory.  S and the weights are double-buffered: a tile's softmax runs while the tile before it is
// multiplied.  `gate` (or null): the output is multiplied by sigmoid(gate) on its way out.
// Every wait is bounded; one that gives up sets the status word and an abort flag, and the CTA frees its tensor memory
// and returns.
#define LE_ROWS 128
#define LE_KEYS 64
#define LE_STAGES 2
#define LE_THREADS 352
#define LE_Q_BOX (LE_ROWS * 128)
#define LE_K_BOX (LE_KEYS * 128)
#define LE_TMEM 256                                                // S twice (64 columns each), PV (at most 128)

struct LatentExpandedArgs {
    const bf16* gate; bf16* out;
    const int* cu_rows; const int* seg_pos; const int* tile_seg; const int* tile_row0; const int* ctx_base;
    int ldo, ldg, rankp, dimp, rotp, vdimp, v_col;
    float scale;
};

__global__ void __launch_bounds__(LE_THREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmE, const __grid_constant__ CUtensorMap tmR,
                         const LatentExpandedArgs p) {
    extern __shared__ unsigned char le_raw[];
    unsigned char* sm = le_raw + ((1024u - (kp_smem_u32(le_raw) & 1023u)) & 1023u);
    const int nb = (p.dimp + 63) >> 6, rb = (p.rotp + 63) >> 6, vb = (p.vdimp + 63) >> 6;      // boxes of the three parts
    const uint32_t stage_bytes = (uint32_t)(nb + rb + vb) * LE_K_BOX;
    unsigned char* Qs = sm;                                        // [nb + rb][128 rows x 128 bytes]
    unsigned char* St = Qs + (size_t)(nb + rb) * LE_Q_BOX;         // [LE_STAGES][nb + rb + vb][64 rows x 128 bytes]
    unsigned char* Ps = St + LE_STAGES * stage_bytes;              // [2][3 parts][128 rows x 128 bytes]
    uint64_t* bars = reinterpret_cast<uint64_t*>(Ps + 2 * 3 * LE_Q_BOX);
    uint64_t* q_full = bars;
    uint64_t* k_full = bars + 1;                                   // [LE_STAGES]
    uint64_t* k_empty = k_full + LE_STAGES;                        // [LE_STAGES]
    uint64_t* s_full = k_empty + LE_STAGES;                        // [2]
    uint64_t* p_full = s_full + 2;                                 // [2]
    uint64_t* o_full = p_full + 2;
    uint64_t* o_empty = o_full + 1;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_empty + 1);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        kp_mbar_init(q_full, 1);
        for (int s = 0; s < LE_STAGES; s++) { kp_mbar_init(&k_full[s], 1); kp_mbar_init(&k_empty[s], 1); }
        for (int b = 0; b < 2; b++) { kp_mbar_init(&s_full[b], 1); kp_mbar_init(&p_full[b], 256); }
        kp_mbar_init(o_full, 1);
        kp_mbar_init(o_empty, 8);
        *abort_flag = 0;
        kp_mbar_init_fence();
    }
    if (warp == 1) kp_tmem_alloc(tmem_slot, LE_TMEM);
    kp_tc_fence_before();
    __syncthreads();
    kp_tc_fence_after();
    const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 2 * LE_KEYS;
    kp_pdl_begin();
    const int h = blockIdx.y, seg = p.tile_seg[blockIdx.x], row0 = p.tile_row0[blockIdx.x];
    const int n_rows = min(LE_ROWS, p.cu_rows[seg + 1] - row0);
    const int pos0 = p.seg_pos[seg] + (row0 - p.cu_rows[seg]);
    const int k_hi = pos0 + n_rows - 1, n_kt = k_hi / LE_KEYS + 1;
    const int Dq = p.dimp + p.rotp;

    if (warp == 0) {
        if (lane == 0) {
            const int base = p.ctx_base[seg];
            kp_mbar_expect_tx(q_full, (uint32_t)(nb + rb) * LE_Q_BOX);
            for (int j = 0; j < nb; j++) kp_tma_load_2d(Qs + (size_t)j * LE_Q_BOX, &tmQ, h * Dq + j * 64, row0, q_full);
            for (int j = 0; j < rb; j++) kp_tma_load_2d(Qs + (size_t)(nb + j) * LE_Q_BOX, &tmQ, h * Dq + p.dimp + j * 64, row0, q_full);
            for (int kt = 0; kt < n_kt; kt++) {
                const int s = kt % LE_STAGES;
                if (*abort_flag || !kp_mbar_wait_bounded(&k_empty[s], ((kt / LE_STAGES) & 1) ^ 1)) { *abort_flag = 1; break; }
                unsigned char* st = St + (size_t)s * stage_bytes;
                const int y = base + kt * LE_KEYS;
                kp_mbar_expect_tx(&k_full[s], stage_bytes);
                for (int j = 0; j < nb; j++) kp_tma_load_2d(st + (size_t)j * LE_K_BOX, &tmE, h * p.dimp + j * 64, y, &k_full[s]);
                for (int j = 0; j < rb; j++) kp_tma_load_2d(st + (size_t)(nb + j) * LE_K_BOX, &tmR, p.rankp + j * 64, y, &k_full[s]);
                for (int j = 0; j < vb; j++)
                    kp_tma_load_2d(st + (size_t)(nb + rb + j) * LE_K_BOX, &tmE, p.v_col + h * p.vdimp + j * 64, y, &k_full[s]);
            }
        }
    } else if (warp == 1) {
        constexpr uint32_t idesc = kp_umma_idesc(LE_ROWS, LE_KEYS);
        const uint64_t q_desc = kp_umma_desc(kp_smem_u32(Qs)), k_desc = kp_umma_desc(kp_smem_u32(St));
        const int n_d = p.dimp >> 4, n_r = p.rotp >> 4;            // steps of 16 columns
        bool ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(q_full, 0));
        for (int kt = 0; kt < n_kt && ok; kt++) {
            const int s = kt % LE_STAGES;
            ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(&k_full[s], (kt / LE_STAGES) & 1));
            if (ok && kt > 1) ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(&p_full[kt & 1], ((kt - 2) >> 1) & 1));
            if (!ok || __any_sync(0xffffffffu, *abort_flag)) { ok = false; break; }
            kp_tc_fence_after();
            const uint64_t kd = k_desc + s * (stage_bytes >> 4);
            const uint32_t d = tmem_s + (kt & 1) * LE_KEYS;
            for (int k = 0; k < n_d; k++)
                kp_umma_bf16_warp(d, q_desc + (k >> 2) * (LE_Q_BOX >> 4) + 2 * (k & 3), kd + (k >> 2) * (LE_K_BOX >> 4) + 2 * (k & 3), idesc, k ? 1u : 0u);
            for (int k = 0; k < n_r; k++)
                kp_umma_bf16_warp(d, q_desc + (nb + (k >> 2)) * (LE_Q_BOX >> 4) + 2 * (k & 3), kd + (nb + (k >> 2)) * (LE_K_BOX >> 4) + 2 * (k & 3),
                                  idesc, 1u);
            kp_umma_commit_warp(&s_full[kt & 1]);
        }
        if (!ok) *abort_flag = 1;
    } else if (warp == 10) {
        const uint32_t idesc = kp_umma_idesc(LE_ROWS, p.vdimp, true);
        const uint64_t p_desc = kp_umma_desc(kp_smem_u32(Ps)), v_desc = kp_umma_desc_mn(kp_smem_u32(St) + (nb + rb) * LE_K_BOX, LE_K_BOX);
        bool ok = true;
        for (int kt = 0; kt < n_kt && ok; kt++) {
            const int s = kt % LE_STAGES;
            ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(&p_full[kt & 1], (kt >> 1) & 1));
            if (ok && kt > 0) ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(o_empty, (kt - 1) & 1));
            if (!ok || __any_sync(0xffffffffu, *abort_flag)) { ok = false; break; }
            kp_tc_fence_after();
            const uint64_t pd = p_desc + (kt & 1) * (3 * LE_Q_BOX >> 4), vd = v_desc + s * (stage_bytes >> 4);
            for (int part = 0; part < 3; part++) {
#pragma unroll
                for (int kk = 0; kk < LE_KEYS / 16; kk++)
                    kp_umma_bf16_warp(tmem_o, pd + part * (LE_Q_BOX >> 4) + 2 * kk, vd + kk * (2048 >> 4), idesc, (part | kk) ? 1u : 0u);
            }
            kp_umma_commit_warp(o_full);
            kp_umma_commit_warp(&k_empty[s]);
        }
        if (!ok) *abort_flag = 1;
    } else {
        const int grp = (warp - 2) >> 2, q4 = warp & 3, r = q4 * 32 + lane;            // r: this thread's row
        const uint32_t lane_off = (uint32_t)(q4 * 32) << 16;
        const int pos = pos0 + r, vh = p.vdimp >> 1;               // the thread's value columns: vh from grp * vh on
        const float sl2 = p.scale * 1.4426950408889634f;
        float acc[64];
#pragma unroll
        for (int i = 0; i < 64; i++) acc[i] = 0.f;
        float m = -INFINITY, l = 0.f, corr_next = 0.f;
        bool ok = true;
        auto softmax = [&](int kt) {
            const int b = kt & 1;
            if (ok) ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(&s_full[b], (kt >> 1) & 1) && !*abort_flag);    // (a warp gives up as one)
            if (!ok) return;
            kp_tc_fence_after();
            const uint32_t ts = tmem_s + b * LE_KEYS + lane_off;
            const int k0 = kt * LE_KEYS;
            uint32_t mine[32];
            float mx = -INFINITY;
            {
                uint32_t other[32];
                kp_tmem_ld32_issue(ts + (grp ^ 1) * 32, other);
                kp_tmem_ld32_issue(ts + grp * 32, mine);
                kp_tmem_ld_wait();
                if (k0 + LE_KEYS - 1 > pos0) {                     // the tile reaches beyond the first row's position
#pragma unroll
                    for (int j = 0; j < 32; j++) {
                        if (k0 + (grp ^ 1) * 32 + j <= pos) mx = fmaxf(mx, __uint_as_float(other[j]));
                        if (k0 + grp * 32 + j > pos) mine[j] = 0xff800000u;                 // -inf
                        mx = fmaxf(mx, __uint_as_float(mine[j]));
                    }
                } else {
#pragma unroll
                    for (int j = 0; j < 32; j++) mx = fmaxf(mx, fmaxf(__uint_as_float(other[j]), __uint_as_float(mine[j])));
                }
            }
            if (kt == n_kt - 1 && k_hi + 1 - k0 < LE_KEYS) {
                // the last tile: values of keys behind the context (another request's, or nobody's) meet weights of 0 and are
                // cleared (0 times NaN is not 0)
                const int first = k_hi + 1 - k0;
                unsigned char* vt = St + (size_t)(kt % LE_STAGES) * stage_bytes + (size_t)(nb + rb) * LE_K_BOX;
                for (int i = threadIdx.x - 64; i < (LE_KEYS - first) * vb * 8; i += 256)
                    *reinterpret_cast<uint4*>(vt + (size_t)((i >> 3) % vb) * LE_K_BOX + (first + (i >> 3) / vb) * 128 + (i & 7) * 16) = make_uint4(0, 0, 0, 0);
            }
            const float m_new = fmaxf(m, mx * sl2);                // (finite: every row sees key 0)
            corr_next = la_exp2(m - m_new);
            m = m_new;
            unsigned char* pr = Ps + (size_t)b * 3 * LE_Q_BOX + r * 128;
            float sum = 0.f;
#pragma unroll
            for (int c = 0; c < 4; c++) {                          // eight keys: a 16-byte piece of the row in each part
                float w[8];
#pragma unroll
                for (int j = 0; j < 8; j++) { w[j] = la_exp2(fmaf(__uint_as_float(mine[c * 8 + j]), sl2, -m_new)); sum += w[j]; }
                const int piece = ((grp * 4 + c) ^ (r & 7)) << 4;
#pragma unroll
                for (int part = 0; part < 3; part++) {
                    uint4 o;
                    o.x = pack_bf16_part(w[0], w[1]); o.y = pack_bf16_part(w[2], w[3]);
                    o.z = pack_bf16_part(w[4], w[5]); o.w = pack_bf16_part(w[6], w[7]);
                    *reinterpret_cast<uint4*>(pr + (size_t)part * LE_Q_BOX + piece) = o;
                }
            }
            l = fmaf(l, corr_next, sum);
            kp_tc_fence_before();                                  // the reads of S are done
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // the weights are read by the tensor core
            kp_mbar_arrive(&p_full[b]);
        };
        softmax(0);
        for (int kt = 0; kt < n_kt && ok; kt++) {
            const float corr = corr_next;
            if (kt + 1 < n_kt) softmax(kt + 1);
            if (ok) ok = __all_sync(0xffffffffu, kp_mbar_wait_bounded(o_full, kt & 1) && !*abort_flag);
            if (!ok) break;
            kp_tc_fence_after();
#pragma unroll
            for (int c = 0; c < 4; c += 2) {
                if (c * 16 < vh) {
                    uint32_t u[2][16];
                    kp_tmem_ld16_issue(tmem_o + lane_off + grp * vh + c * 16, u[0]);
                    if ((c + 1) * 16 < vh) kp_tmem_ld16_issue(tmem_o + lane_off + grp * vh + (c + 1) * 16, u[1]);
                    kp_tmem_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; i++) acc[c * 16 + i] = fmaf(acc[c * 16 + i], corr, __uint_as_float(u[0][i]));
                    if ((c + 1) * 16 < vh) {
#pragma unroll
                        for (int i = 0; i < 16; i++) acc[c * 16 + 16 + i] = fmaf(acc[c * 16 + 16 + i], corr, __uint_as_float(u[1][i]));
                    }
                }
            }
            kp_tc_fence_before();
            __syncwarp();
            if (lane == 0) kp_mbar_arrive(o_empty);
        }
        if (!ok) *abort_flag = 1;
        // the two threads of a row put their sums together (every product has read Q by now: its place takes them)
        float* sums = reinterpret_cast<float*>(Qs);
        sums[grp * LE_ROWS + r] = l;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (ok && r < n_rows) {
            const float inv = 1.0f / (sums[r] + sums[LE_ROWS + r]);
            const size_t col = (size_t)h * p.vdimp + grp * vh;
            bf16* dst = p.out + (size_t)(row0 + r) * p.ldo + col;
            const bf16* g = p.gate ? p.gate + (size_t)(row0 + r) * p.ldg + col : nullptr;
#pragma unroll
            for (int c = 0; c < 64; c += 8) {
                if (c < vh) {
                    float f[8];
#pragma unroll
                    for (int i = 0; i < 8; i++) f[i] = acc[c + i] * inv;
                    if (g) {
                        const uint4 raw = *reinterpret_cast<const uint4*>(g + c);
                        const __nv_bfloat162* z2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            const float2 z = __bfloat1622float2(z2[i]);
                            f[2 * i] /= 1.0f + expf(-z.x);
                            f[2 * i + 1] /= 1.0f + expf(-z.y);
                        }
                    }
                    uint4 o;
                    o.x = pack_bf16(f[0], f[1]); o.y = pack_bf16(f[2], f[3]); o.z = pack_bf16(f[4], f[5]); o.w = pack_bf16(f[6], f[7]);
                    *reinterpret_cast<uint4*>(dst + c) = o;
                }
            }
        }
    }
    kp_tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        if (threadIdx.x == 0) atomicExch(&g_latent_status, 1);
        kp_linger_after_failure();
    }
    if (warp == 1) kp_tmem_dealloc(tmem_s, LE_TMEM);
}

static size_t le_smem(int dimp, int rotp, int vdimp) {
    const int nb = (dimp + 63) / 64, rb = (rotp + 63) / 64, vb = (vdimp + 63) / 64;
    return 1024 + (size_t)(nb + rb) * LE_Q_BOX + (size_t)LE_STAGES * (nb + rb + vb) * LE_K_BOX + 6 * LE_Q_BOX + (2 * LE_STAGES + 7) * 8 + 16;
}

static size_t lt_fixed_bytes(int n_box, int nh) {
    return 1024 + (size_t)n_box * nh * 128 + 2 * 3 * nh * 128 + 16 * nh * sizeof(float) + (2 * LT_MAX_STAGES + 7) * 8 + 16;
}
#define LT_SMEM_MAX (226 * 1024)

// Can the tensor-core form of the absorbed pass take these sizes (two tiles in shared memory, the latent's blocks in tensor
// memory, pages that boxes of rows divide)?
static bool lt_fits(int rankp, int W, int H, int page_size) {
    const int n_box = W / 64;
    return rankp <= 512 && W % 64 == 0 && page_size % 8 == 0 && (page_size % LT_TILE == 0 || LT_TILE % page_size == 0) &&
           lt_fixed_bytes(n_box, H > 16 ? 32 : 16) + (size_t)2 * n_box * LT_BOX_BYTES <= LT_SMEM_MAX;
}

template <typename F>
static int la_set_smem(F kern, size_t sm) {
    if (sm <= 48 * 1024) return 0;
    return (int)cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
}

extern "C" {

int kp_latent_prep(void* p, int ld, int q_col, int c_col, int H, int dimp, int rotp, int rank, int rankp, int W, const float* w, float eps,
                   const float* cos_tab, const float* sin_tab, int rot, int interleaved, const int* positions, const int* slot_map,
                   void* cache, int page_size, void* qa, int n_absorbed, int n, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (H < 1 || rank < 1 || rank > rankp || (rankp & 15) || (rotp & 15) || rotp < 0 || W < rankp + rotp || page_size < 1 || (cos_tab && (rot < 2 || (rot & 1) || rot > rotp)) ||
        n_absorbed < 0 || n_absorbed > n || (n_absorbed > 0 && !qa))
        return KP_ERR_BAD_ARG;
    const int groups = H * (rotp >> 3);
    if (dtype == KP_DTYPE_BF16 && (!cos_tab || (interleaved && (rot & 7) == 0)) && !(ld & 7) && !(q_col & 7) && !(c_col & 7) && !(W & 7) && W <= 2048 &&
        groups <= 8 * 256 && !(((uintptr_t)p | (uintptr_t)cache | (uintptr_t)qa | (uintptr_t)cos_tab | (uintptr_t)sin_tab) & 15)) {
#define PREP_VEC(PER)                                                                                                     \
    kp_launch_pdl(latent_prep_vec_kernel<PER>, dim3(n), dim3(256), 0, (cudaStream_t)stream, (bf16*)p, ld, q_col, c_col, H, dimp, rotp, rank, \
                  rankp, W, w, eps, cos_tab, sin_tab, rot, positions, slot_map, (bf16*)cache, page_size, (bf16*)qa, n_absorbed)
        if (groups <= 256) PREP_VEC(1); else if (groups <= 512) PREP_VEC(2); else if (groups <= 1024) PREP_VEC(4); else PREP_VEC(8);
#undef PREP_VEC
        return kp_launch_status();
    }
    KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(latent_prep_kernel<T>, dim3(n), dim3(256), 0, (cudaStream_t)stream, (T*)p, ld, q_col, c_col, H,
                                               dimp, rotp, rank, rankp, W, w, eps, cos_tab, sin_tab, rot, interleaved, positions,
                                               slot_map, (T*)cache, page_size, (T*)qa, n_absorbed)));
    return kp_launch_status();
}

// out[m, h, :N] = a[m, h, :K] b[h]^T, b [H][N][K]; strides in elements.  N and K multiples of 16.
int kp_head_gemm(const void* a, long long a_row, int a_head, const void* b, void* out, long long o_row, int o_head, const void* gate,
                 long long g_row, int g_head, int M, int N, int K, int H, int dtype, void* stream) {
    if (M <= 0) return 0;
    if (N < 1 || K < 1 || H < 1 || (N & 15) || (K & 15) || H > 65535) return KP_ERR_BAD_ARG;
    HeadGemmArgs p = {a, b, gate, out, a_row, o_row, g_row, a_head, o_head, g_head, M, N, K, H};
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == KP_DTYPE_BF16 && !(((uintptr_t)a | (uintptr_t)b | (uintptr_t)out) & 15) && !(a_row & 7) && !(a_head & 7) && !(o_row & 1) &&
        !(o_head & 1) && (!gate || (!((uintptr_t)gate & 3) && !(g_row & 1) && !(g_head & 1)))) {
        const int gx = (N + 31) / 32;
        if (M <= 16) kp_launch_pdl(head_gemm_mma_kernel<1>, dim3(gx, H, 1), dim3(128), 0, s, p);
        else if (M <= 32) kp_launch_pdl(head_gemm_mma_kernel<2>, dim3(gx, H, 1), dim3(128), 0, s, p);
        else kp_launch_pdl(head_gemm_mma_kernel<4>, dim3(gx, H, (M + 63) / 64), dim3(128), 0, s, p);
        return kp_launch_status();
    }
    KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(head_gemm_simt_kernel<T>, dim3((N + 63) / 64, H, (M + 15) / 16), dim3(256), 0, s, p)));
    return kp_launch_status();
}

// The chunks a row has at most in kp_latent_split with these sizes (its scratch: n H chunks (rankp + 2) floats).  The tensor-core
// form: as many as give the fewest rounds of CTAs over the SMs (one an SM) times the tiles of a CTA, what a CTA
// costs beside its tiles (launch, the first tile's way, the last one's products: about two and a half tiles) counted in.
int kp_latent_chunks(int n, int max_context, int rankp, int W, int H, int page_size, int dtype, int tensor_cores) {
    if (!(tensor_cores && dtype == KP_DTYPE_BF16 && lt_fits(rankp, W, H, page_size))) return (max_context + LA_CHUNK - 1) / LA_CHUNK;
    const long long ctas = (long long)n * ((H + (H > 16 ? 31 : 15)) / (H > 16 ? 32 : 16));
    const int tiles = (max_context + LT_TILE - 1) / LT_TILE, sms = 148;
    int best_c = 1;
    double best = 1e30;
    for (int c = 1; c <= tiles && c <= 512; c++) {
        const double cost = (double)((ctas * c + sms - 1) / sms) * ((tiles + c - 1) / c + 2.5);
        if (cost < best) { best = cost; best_c = c; }
    }
    return best_c;
}

// qa [n][H][W] -> u [n][H][rankp]; max_context: beyond the largest position of the rows; n_pages: pages of the cache.
int kp_latent_split(const void* qa, const void* cache, long long n_pages, const int* block_table, int max_blocks, const int* row_seg,
                    const int* positions, float* scratch, int max_context, void* u, float scale, int page_size, int n, int H, int rankp,
                    int W, int dtype, int tensor_cores, void* stream) {
    if (n <= 0) return 0;
    if (n > 65535 || H < 1 || max_context < 1 || page_size < 1 || (rankp & 15) || (W & 15) || rankp < 16 || W < rankp)
        return KP_ERR_BAD_ARG;
    const int n_chunks = kp_latent_chunks(n, max_context, rankp, W, H, page_size, dtype, tensor_cores);
    float* part_acc = scratch;
    float* part_ml = scratch + (size_t)n * H * n_chunks * rankp;
    cudaStream_t s = (cudaStream_t)stream;
    int st = 0;
    const bool tc = tensor_cores && dtype == KP_DTYPE_BF16 && lt_fits(rankp, W, H, page_size);
    if (tc) {
        if (((uintptr_t)qa | (uintptr_t)cache) & 15 || n_pages * page_size >= 2147483647LL || (long long)n * H >= 2147483647LL) return KP_ERR_UNSUPPORTED;
        const int nh = H > 16 ? 32 : 16, n_box = W / 64;
        const size_t fixed = lt_fixed_bytes(n_box, nh), tile = (size_t)n_box * LT_BOX_BYTES;
        int stages = (int)((LT_SMEM_MAX - fixed) / tile);
        if (stages > LT_MAX_STAGES) stages = LT_MAX_STAGES;
        const size_t sm = fixed + stages * tile;
        alignas(64) CUtensorMap tc_map, tq_map;
        st = page_size < LT_TILE ? kp_make_map_bf16_groups(&tc_map, cache, (unsigned long long)n_pages * page_size, n_box, W, page_size, 1)
                                 : kp_make_map_bf16_groups(&tc_map, cache, (unsigned long long)n_pages * page_size, n_box, W, LT_TILE);
        if (!st) st = kp_make_map_bf16_groups(&tq_map, qa, (unsigned long long)n * H, n_box, W, nh);
        if (st) return st;
        LatentSplitArgs a = {block_table, row_seg, positions, part_acc, part_ml, max_blocks, n_chunks, page_size, H, rankp, n_box, stages, scale};
        dim3 grid(n_chunks, (H + nh - 1) / nh, n);
        auto kern = nh == 16 ? latent_split_tc_kernel<16> : latent_split_tc_kernel<32>;
        st = la_set_smem(kern, sm);
        if (st) return st;
        kp_launch_pdl(kern, grid, dim3(LT_THREADS), sm, s, tc_map, tq_map, a);
    } else {
        const size_t sm = ((size_t)LA_SCALAR_HEADS * (W + LA_CHUNK) + 32 + LA_CHUNK) * sizeof(float);
        if (sm > 200 * 1024) return KP_ERR_UNSUPPORTED;
        dim3 grid(n_chunks, (H + LA_SCALAR_HEADS - 1) / LA_SCALAR_HEADS, n);
        KP_DISPATCH_DTYPE(dtype, T, {
            st = la_set_smem(latent_split_kernel<T>, sm);
            if (st) return st;
            kp_launch_pdl(latent_split_kernel<T>, grid, dim3(LA_CHUNK), sm, s, (const T*)qa, (const T*)cache, block_table, max_blocks, row_seg,
                          positions, part_acc, part_ml, n_chunks, scale, page_size, H, rankp, W);
        });
    }
    st = kp_launch_status();
    if (st) return st;
    const size_t msm = ((size_t)n_chunks + 32) * sizeof(float);
    if (msm > 200 * 1024) return KP_ERR_UNSUPPORTED;
    KP_DISPATCH_DTYPE(dtype, T, {
        st = la_set_smem(latent_merge_kernel<T>, msm);
        if (st) return st;
        kp_launch_pdl(latent_merge_kernel<T>, dim3(H, n), dim3(128), msm, s, part_acc, part_ml, positions, (T*)u, n_chunks, H, rankp,
                      tc ? 0 : 1);
    });
    return kp_launch_status();
}

int kp_latent_gather(const void* cache, const int* block_table, int max_blocks, const int* ctx_base, int n_seg, void* out, int n_rows,
                     int page_size, int W, void* stream) {
    if (n_rows <= 0) return 0;
    if (n_seg < 1 || page_size < 1 || (W & 7)) return KP_ERR_BAD_ARG;
    kp_launch_pdl(latent_gather_kernel, dim3((n_rows + 7) / 8), dim3(256), 0, (cudaStream_t)stream, (const bf16*)cache, block_table, max_blocks,
                  ctx_base, n_seg, (bf16*)out, n_rows, page_size, W);
    return kp_launch_status();
}

// 1 if the tcgen05 form of the expanded pass takes these sizes.
int kp_latent_prefill_tc_ok(int dimp, int rotp, int vdimp) {
    return !(dimp & 15) && !(rotp & 15) && dimp >= 16 && rotp >= 16 && vdimp >= 32 && vdimp % 32 == 0 && vdimp <= 128 &&
           le_smem(dimp, rotp, vdimp) <= LT_SMEM_MAX;
}

// As kp_latent_prefill, with tiles of 128 rows, on the tcgen05 tensor cores; n_rows rows of q, n_ctx rows of ex and `rows`; gate
// (rows ldg apart, H heads of vdimp) or null: the output times sigmoid(gate).
int kp_latent_prefill_tc(const void* q, int ldq, int n_rows, const void* ex, int ld_ex, int v_col, const void* rows, int n_ctx, int W, int rankp,
                         int dimp, int rotp, int vdimp, const int* cu_rows, const int* seg_pos, const int* tile_seg, const int* tile_row0,
                         const int* ctx_base, int n_tiles, const void* gate, int ldg, void* out, int ldo, float scale, int H, void* stream) {
    if (n_tiles <= 0) return 0;
    if (!kp_latent_prefill_tc_ok(dimp, rotp, vdimp) || (rankp & 15) || W < rankp + rotp || H < 1 || H > 65535 || n_rows < 1 || n_ctx < 1)
        return KP_ERR_BAD_ARG;
    if ((ldq & 7) || (ldo & 7) || (ld_ex & 7) || (v_col & 7) || (W & 7) || (gate && (ldg & 7)) ||
        (((uintptr_t)q | (uintptr_t)ex | (uintptr_t)rows | (uintptr_t)out | (uintptr_t)gate) & 15))
        return KP_ERR_UNSUPPORTED;
    alignas(64) CUtensorMap tq, te, tr;
    int st = kp_make_map_bf16_2d(&tq, q, (unsigned long long)n_rows, H * (dimp + rotp), ldq, 64, LE_ROWS);
    if (!st) st = kp_make_map_bf16_2d(&te, ex, (unsigned long long)n_ctx, v_col + H * vdimp, ld_ex, 64, LE_KEYS);
    if (!st) st = kp_make_map_bf16_2d(&tr, rows, (unsigned long long)n_ctx, W, W, 64, LE_KEYS);
    if (st) return st;
    const size_t sm = le_smem(dimp, rotp, vdimp);
    st = la_set_smem(latent_prefill_tc_kernel, sm);
    if (st) return st;
    LatentExpandedArgs a = {(const bf16*)gate, (bf16*)out, cu_rows, seg_pos, tile_seg, tile_row0, ctx_base, ldo, ldg, rankp, dimp, rotp, vdimp, v_col, scale};
    kp_launch_pdl(latent_prefill_tc_kernel, dim3(n_tiles, H), dim3(LE_THREADS), sm, (cudaStream_t)stream, tq, te, tr, a);
    return kp_launch_status();
}

// q: rows of H heads of dimp + rotp; ex [T][ld_ex]: the expanded keys (H heads of dimp) and, from v_col on, values (H
// heads of vdimp); rows [T][W]: the gathered cache rows; tile_seg / tile_row0: n_tiles tiles of 64 rows.
int kp_latent_prefill(const void* q, int ldq, const void* ex, int ld_ex, int v_col, const void* rows, int W, int rankp, int dimp, int rotp,
                      int vdimp, const int* cu_rows, const int* seg_pos, const int* tile_seg, const int* tile_row0, const int* ctx_base,
                      int n_tiles, void* out, int ldo, float scale, int H, void* stream) {
    if (n_tiles <= 0) return 0;
    if ((dimp & 15) || (rotp & 15) || (vdimp & 15) || (rankp & 15) || (W & 7) || W < rankp + rotp || H < 1 || H > 65535) return KP_ERR_BAD_ARG;
    if ((ldq & 1) || (ldo & 1) || (ld_ex & 7) || (v_col & 7) || (((uintptr_t)ex | (uintptr_t)rows) & 15)) return KP_ERR_UNSUPPORTED;
    const int Dq = dimp + rotp;
    LatentPrefillArgs a = {(const bf16*)q, (const bf16*)ex, (const bf16*)rows, (bf16*)out, cu_rows, seg_pos, tile_seg, tile_row0, ctx_base,
                           ldq, ldo, ld_ex, W, rankp, dimp, rotp, vdimp, v_col, n_tiles, scale};
    const size_t sm = (size_t)2 * LP_TILE * (Dq + 8 + vdimp + 8) * 2;
    if (sm > 200 * 1024) return KP_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    int st;
#define LP_LAUNCH(KS, VT)                                                                                                 \
    do {                                                                                                                  \
        st = la_set_smem(latent_prefill_kernel<KS, VT>, sm);                                                              \
        if (st) return st;                                                                                                \
        kp_launch_pdl(latent_prefill_kernel<KS, VT>, dim3(n_tiles, H), dim3(128), sm, s, a);                              \
        return kp_launch_status();                                                                                        \
    } while (0)
    if (Dq <= 128 && vdimp <= 64) LP_LAUNCH(8, 8);
    if (Dq <= 128 && vdimp <= 128) LP_LAUNCH(8, 16);
    if (Dq <= 192 && vdimp <= 128) LP_LAUNCH(12, 16);
    if (Dq <= 256 && vdimp <= 256) LP_LAUNCH(16, 32);
#undef LP_LAUNCH
    return KP_ERR_UNSUPPORTED;
}

}  // extern "C"
