// Causal GQA attention of a batch of rows over the paged cache.
//
// For the row at position p of a request, head h reads kv head g = h / (H/G)
// and the keys t in [max(0, p - window + 1), p] (window <= 0: all keys):
//   s_t = (q . K_t) * scale ;  out = sum_t softmax(s)_t V_t
// Two variants, each an argument: `keep_first` > 0 lets every row also read the keys 0 .. keep_first - 1 that
// lie before its window (at their true places: the tiles between them and the window are skipped); `sink`
// (one float32 number a query head, or null) adds exp(sink_h) to the softmax's denominator, a key that has a
// score but no value, counted once a row.
// Three more: `cap` > 0 bounds the scores, s <- cap tanh(s / cap); `pool` > 0 (with a window): the row also reads one
// key and value for each block of `pool` positions that lies wholly before its window, the blocks' means as another
// kernel left them in a cache of their own (entry b of the request's pooled block table); `out_scale` multiplies the
// output.
// (src/backend/cpu/scalar/core.c:383-433: online softmax with running max M,
// sum S and rescaled accumulator).  Keys are found through the request's
// block table: key t lies in page table[t / page_size] at offset t % page_size
// of the layer's cache [page][K|V][G][page_size][hd].  The keys of the rows of
// this very step were written before this kernel runs, so a prompt portion
// sees the earlier pages and its own rows alike.
//
// General kernel (any head_dim that is a multiple of 2 up to 256, any H, G,
// page size, window): one block per (head, row), 128 keys per tile, float32
// statistics.  Tiles start at multiples of 128 of the absolute key index, so
// the order of summation does not depend on how a prompt was cut.
#include "common.cuh"

#define ATT_THREADS 128
#define KP_MAX_HEAD_DIM 256

template <typename T>
__global__ void __launch_bounds__(ATT_THREADS)
attention_rows_kernel(const T* __restrict__ q, int ldq, const T* __restrict__ cache,
                      const int* __restrict__ block_table, int max_blocks, const int* __restrict__ row_seg,
                      const int* __restrict__ positions, T* __restrict__ out, int ldo, float scale, int window,
                      int page_size, int H, int G, int hd, int block, int keep_first, const float* __restrict__ sink, float cap,
                      float out_scale, int pool, const T* __restrict__ pool_cache, const int* __restrict__ pool_table, int max_pool_blocks) {
    kp_pdl_begin();
    __shared__ float qs[KP_MAX_HEAD_DIM];
    __shared__ float ps[ATT_THREADS];
    __shared__ float red[32];
    const int tid = threadIdx.x;
    const int h = blockIdx.x, row = blockIdx.y;
    const int g = h / (H / G);
    const int pos = positions[row];
    const int* bt = block_table + (size_t)row_seg[row] * max_blocks;
    int k_lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (block > 0) k_lo = max(k_lo, (pos / block) * block);      // nothing from before the row's own block of positions
    const int k_hi = pos;
    const int first_hi = min(keep_first, k_lo);                  // keys 0 .. first_hi - 1 are read as well
    const size_t page_stride = (size_t)2 * G * page_size * hd;   // elements per page (K and V)
    const size_t k_off = (size_t)g * page_size * hd;
    const size_t v_off = ((size_t)G + g) * page_size * hd;

    for (int i = tid; i < hd; i += ATT_THREADS) qs[i] = to_f32(q[(size_t)row * ldq + (size_t)h * hd + i]);
    __syncthreads();

    // (the sink enters as a key that was seen before all others: maximum sink_h, sum 1, no value)
    float m = sink ? sink[h] : -INFINITY, l = sink ? 1.f : 0.f;
    float acc0 = 0.f, acc1 = 0.f;
    // (the pooled entries come first, in tiles of their own from 0 on; the tokens' tiles follow)
    const int n_pool = pool > 0 ? kp_pooled_count(pos, window, pool) : 0;
    const int* pt = pool > 0 ? pool_table + (size_t)row_seg[row] * max_pool_blocks : nullptr;
    for (int pass = n_pool > 0 ? 0 : 1; pass < 2; pass++) {
    const int* tab = pass == 0 ? pt : bt;
    const T* kv = pass == 0 ? pool_cache : cache;
    const int r_lo = pass == 0 ? 0 : k_lo, r_hi = pass == 0 ? n_pool - 1 : k_hi, first = pass == 0 ? 0 : first_hi;
    for (int tile0 = first > 0 ? 0 : (r_lo / ATT_THREADS) * ATT_THREADS; tile0 <= r_hi; tile0 += ATT_THREADS) {
        if (tile0 >= first && tile0 + ATT_THREADS <= r_lo) {  // between the kept keys and the window: on to the window's tile
            tile0 = (r_lo / ATT_THREADS) * ATT_THREADS - ATT_THREADS;
            continue;
        }
        const int key = tile0 + tid;
        const bool valid = key <= r_hi && (key >= r_lo || key < first);
        float s = -INFINITY;
        if (valid) {
            const T* kp = kv + (size_t)tab[key / page_size] * page_stride + k_off + (size_t)(key % page_size) * hd;
            float dot = 0.f;
            for (int i = 0; i < hd; i++) dot = fmaf(qs[i], to_f32(kp[i]), dot);
            s = kp_capped(dot * scale, cap);
        }
        const float m_new = fmaxf(m, block_max(s, red));
        const float pe = valid ? expf(s - m_new) : 0.f;
        const float corr = (m == -INFINITY) ? 0.f : expf(m - m_new);
        const float tsum = block_sum(pe, red);
        l = l * corr + tsum;
        __syncthreads();
        ps[tid] = pe;
        __syncthreads();
        acc0 *= corr;
        acc1 *= corr;
        const int kk_hi = min(r_hi - tile0, ATT_THREADS - 1);
        for (int kk = 0; kk <= kk_hi; kk++) {
            const int key2 = tile0 + kk;
            if (key2 < r_lo && key2 >= first) continue;
            const T* vp = kv + (size_t)tab[key2 / page_size] * page_stride + v_off + (size_t)(key2 % page_size) * hd;
            const float pv = ps[kk];
            if (tid < hd) acc0 = fmaf(pv, to_f32(vp[tid]), acc0);
            if (tid + ATT_THREADS < hd) acc1 = fmaf(pv, to_f32(vp[tid + ATT_THREADS]), acc1);
        }
        m = m_new;
    }
    }
    const float inv = l > 0.f ? out_scale / l : 0.f;
    T* o = out + (size_t)row * ldo + (size_t)h * hd;
    if (tid < hd) o[tid] = from_f32<T>(acc0 * inv);
    if (tid + ATT_THREADS < hd) o[tid + ATT_THREADS] = from_f32<T>(acc1 * inv);
}

// block: 0, or the size of the blocks of positions (counted from 0) beyond whose start a row reads no keys.
// keep_first: the first keys of the sequence that stay readable behind a window; sink: [H] float32 or null.
// cap: 0, or the bound of the scores; out_scale: factor of the output; pool: 0, or the positions of a pooled block (then
// pool_cache [pages][K|V][G][page_size][hd] and pool_table [requests][max_pool_blocks] hold the blocks' means).
extern "C" int kp_attention_rows_pooled(const void* q, int ldq, const void* cache, const int* block_table, int max_blocks,
                                        const int* row_seg, const int* positions, void* out, int ldo, float scale,
                                        int window, int block, int keep_first, const float* sink, float cap, float out_scale,
                                        int pool, const void* pool_cache, const int* pool_table, int max_pool_blocks,
                                        int page_size, int n, int H, int G, int hd, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (cap < 0.f || pool < 0 || (pool > 0 && (window <= 0 || block > 0 || keep_first > 0 || !pool_cache || !pool_table)))
        return KP_ERR_BAD_ARG;
    if (keep_first < 0 || (keep_first > 0 && block > 0)) return KP_ERR_BAD_ARG;
    if (hd < 2 || hd > KP_MAX_HEAD_DIM) return KP_ERR_UNSUPPORTED;
    if (G < 1 || H % G != 0 || page_size < 1) return KP_ERR_BAD_ARG;
    if (n > 65535) return KP_ERR_UNSUPPORTED;
    dim3 grid(H, n);
    KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(attention_rows_kernel<T>, dim3(grid), dim3(ATT_THREADS), 0, (cudaStream_t)stream, 
        (const T*)q, ldq, (const T*)cache, block_table, max_blocks, row_seg, positions, (T*)out, ldo, scale, window,
        page_size, H, G, hd, block, window > 0 ? keep_first : 0, sink, cap, out_scale, pool, (const T*)pool_cache, pool_table,
        max_pool_blocks)));
    return kp_launch_status();
}

extern "C" int kp_attention_rows_sink(const void* q, int ldq, const void* cache, const int* block_table, int max_blocks,
                                      const int* row_seg, const int* positions, void* out, int ldo, float scale,
                                      int window, int block, int keep_first, const float* sink, int page_size, int n,
                                      int H, int G, int hd, int dtype, void* stream) {
    return kp_attention_rows_pooled(q, ldq, cache, block_table, max_blocks, row_seg, positions, out, ldo, scale, window, block,
                                    keep_first, sink, 0.f, 1.f, 0, nullptr, nullptr, 0, page_size, n, H, G, hd, dtype, stream);
}

extern "C" int kp_attention_rows_masked(const void* q, int ldq, const void* cache, const int* block_table, int max_blocks,
                                        const int* row_seg, const int* positions, void* out, int ldo, float scale,
                                        int window, int block, int page_size, int n, int H, int G, int hd, int dtype,
                                        void* stream) {
    return kp_attention_rows_sink(q, ldq, cache, block_table, max_blocks, row_seg, positions, out, ldo, scale, window, block,
                                  0, nullptr, page_size, n, H, G, hd, dtype, stream);
}

extern "C" int kp_attention_rows(const void* q, int ldq, const void* cache, const int* block_table, int max_blocks,
                                 const int* row_seg, const int* positions, void* out, int ldo, float scale,
                                 int window, int page_size, int n, int H, int G, int hd, int dtype, void* stream) {
    return kp_attention_rows_masked(q, ldq, cache, block_table, max_blocks, row_seg, positions, out, ldo, scale, window, 0,
                                    page_size, n, H, G, hd, dtype, stream);
}
