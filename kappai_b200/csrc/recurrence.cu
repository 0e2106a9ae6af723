// Linear recurrences with data-dependent decays.  A head keeps a float32 state S [D, P] a request and follows, row after
// row,
//
//   F = g S          what is left of the state of the row before
//   e = v            ("gated": gated linear attention), or
//   e = beta (v - F^T k)     ("delta": the gated delta rule: what F holds for k is taken off v first)
//   S' = F + k e^T ,     o = S'^T q ,
//
// g one factor in (0, 1] a head, or one a key channel (a row of S), given by its logarithm.  Several heads may share a
// query and key (head h reads q/k head h / (H / G)).
//
// Everything here is float32: decays and their logarithms, step sizes, unit norms, the state, products and sums; the
// storage type holds projections only.
//
// Kernels: what stands between the projections and a delta recurrence (convolutions over time with silu, unit norms of
// q and k, step sizes, logarithms of decays) in one launch; the logarithms of decays alone for a gated recurrence; the
// scan (row after row, the state in registers, every sum in an order fixed by the sizes alone, so a row's bits do not
// depend on how the sequence was cut); and the chunked form for prompt portions in 16-bit mode (below).
#include "common.cuh"
#include "chanconv.cuh"

// ------------------------------------------------------------------------------------------------ in front of the scan

// The logarithm of a decay from its projection z: kind 0, exp(-A softplus(z + bias)): -A softplus(z + bias), A = exp(A_log);
// kind 1, sigmoid(z)^(1/tau): -softplus(-z) / tau.
__device__ __forceinline__ float rc_log_decay_step(float z, float bias, float neg_a) { return neg_a * ss_softplus(z + bias); }
__device__ __forceinline__ float rc_log_decay_sigmoid(float z, float inv_tau) { return -ss_softplus(-z) * inv_tau; }

// Entry e of a row's H step sizes and its decays (H of them, or H D in place in lg): e < H is beta_e, the rest decays.
template <typename T>
__device__ __forceinline__ void rc_gate_entry(const T* __restrict__ prow, int b_col, int a_col, const float* __restrict__ neg_a,
                                              const float* __restrict__ dt_bias, float* __restrict__ beta, float* __restrict__ lg,
                                              int r, int e, int H, int D, int per_channel) {
    if (e < H) {
        beta[(size_t)r * H + e] = 1.0f / (1.0f + expf(-to_f32(prow[b_col + e])));
        return;
    }
    e -= H;
    if (per_channel) {
        float* z = lg + (size_t)r * H * D + e;
        *z = rc_log_decay_step(*z, dt_bias[e], neg_a[e / D]);
    } else {
        lg[(size_t)r * H + e] = rc_log_decay_step(to_f32(prow[a_col + e]), dt_bias[e], neg_a[e]);
    }
}

// p: rows [n, ld] in the storage type with the channels [q: G heads of D | k: G heads of D | v: H heads of P] side by side
// from conv_col.  out: [n, C] float32, the same channels behind convolution and silu, q and k as unit vectors a head
// (divided by the root of their sum of squares + 1e-6), q times q_scale.  A warp takes one q or k head, or 128 channels of v, or 128 gate entries, of
// one row.  single_rows: every segment has one row, and the lane that read a channel's kept inputs writes the new ones.
#define RP_UNIT_EPS 1e-6f
template <typename T>
__global__ void __launch_bounds__(128)
delta_prep_kernel(const T* __restrict__ p, int ld, int conv_col, int b_col, int a_col, const float* __restrict__ taps,
                  const float* __restrict__ neg_a, const float* __restrict__ dt_bias, float* __restrict__ kept, size_t slot_stride,
                  const int* __restrict__ row_seg, const int* __restrict__ cu_rows, const int* __restrict__ seg_pos,
                  const int* __restrict__ seg_slot, float* __restrict__ out, float* __restrict__ beta, float* __restrict__ lg,
                  int H, int G, int D, int P, int K, float q_scale, int per_channel, int single_rows) {
    kp_pdl_begin();
    const int lane = threadIdx.x & 31;
    int it = blockIdx.x * 4 + (threadIdx.x >> 5);
    const int r = blockIdx.y;
    const int qk = 2 * G, vb = (H * P + 127) / 128, C = 2 * G * D + H * P;
    if (it >= qk + vb) {
        const int e0 = (it - qk - vb) * 128, n_e = H + (per_channel ? H * D : H);
        for (int e = e0 + lane; e < min(e0 + 128, n_e); e += 32)
            rc_gate_entry<T>(p + (size_t)r * ld, b_col, a_col, neg_a, dt_bias, beta, lg, r, e, H, D, per_channel);
        return;
    }
    const int base = it < qk ? it * D : 2 * G * D + (it - qk) * 128;
    const int count = it < qk ? D : min(128, C - base);
    const int seg = row_seg[r], row0 = cu_rows[seg];
    const bool fresh = seg_pos[seg] == 0;
    float* kp = kept + (size_t)seg_slot[seg] * slot_stride;
    // (lane l keeps channels 4 l .. 4 l + 3 where heads are a multiple of 4 wide, so that a head's sum of squares is added in the
    // order of the other form below)
    const bool quads = D % 4 == 0;
    auto place = [&](int j) { return quads ? (j >> 2) * 128 + lane * 4 + (j & 3) : lane + 32 * j; };
    float y[8];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; j++) {
        y[j] = 0.f;
        const int c = base + place(j);
        if (place(j) >= count) continue;
        float acc = 0.f;
        for (int m = 0; m < K; m++) {
            const int rr = r - (K - 1) + m;
            float v;
            if (rr >= row0) v = to_f32(p[(size_t)rr * ld + conv_col + c]);
            else v = fresh ? 0.f : kp[(size_t)(rr - row0 + K - 1) * C + c];
            // (tap m's input becomes the kept input m - 1 of the next row, written behind its read)
            if (single_rows && m > 0) kp[(size_t)(m - 1) * C + c] = v;
            acc = fmaf(taps[(size_t)c * K + m], v, acc);
        }
        y[j] = ss_silu(acc);
        ss = fmaf(y[j], y[j], ss);
    }
    float scale = 1.f;
    if (it < qk) {
        ss = warp_sum(ss);
        scale = 1.0f / sqrtf(ss + RP_UNIT_EPS);
        if (it < G) scale *= q_scale;
    }
    float* dst = out + (size_t)r * C + base;
#pragma unroll
    for (int j = 0; j < 8; j++)
        if (place(j) < count) dst[place(j)] = y[j] * scale;
}

// The same for steps of several rows where heads are multiples of 4 wide and rows start on 8 (16) bytes: a lane takes four
// channels (eight where D > 128: QL = 2) of RP_ROWS consecutive rows and fetches every row of p once for all of them; heads
// of 4, 8, .. 64 channels share a warp.  The blocks from conv_blocks on compute the gate entries of the tile's rows.
#define RP_ROWS 4
__device__ __forceinline__ float4 rp_load4(const float* s) { return __ldg(reinterpret_cast<const float4*>(s)); }
__device__ __forceinline__ float4 rp_load4(const bf16* s) {
    const uint2 raw = __ldg(reinterpret_cast<const uint2*>(s));
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void rp_fma4(float4& acc, const float4 w, const float4 v) {
    acc.x = fmaf(w.x, v.x, acc.x); acc.y = fmaf(w.y, v.y, acc.y); acc.z = fmaf(w.z, v.z, acc.z); acc.w = fmaf(w.w, v.w, acc.w);
}

template <typename T, int K, int QL>
__global__ void __launch_bounds__(128)
delta_prep_vec_kernel(const T* __restrict__ p, int ld, int conv_col, int b_col, int a_col, const float* __restrict__ taps,
                      const float* __restrict__ neg_a, const float* __restrict__ dt_bias, const float* __restrict__ kept,
                      size_t slot_stride, const int* __restrict__ row_seg, const int* __restrict__ cu_rows,
                      const int* __restrict__ seg_pos, const int* __restrict__ seg_slot, float* __restrict__ out,
                      float* __restrict__ beta, float* __restrict__ lg, int n, int H, int G, int D, int P, float q_scale,
                      int per_channel, int conv_blocks, int team) {
    kp_pdl_begin();
    const int r0 = blockIdx.y * RP_ROWS;
    if ((int)blockIdx.x >= conv_blocks) {
        const int n_e = H + (per_channel ? H * D : H);
        for (int i = 0; i < RP_ROWS && r0 + i < n; i++)
            for (int e = (blockIdx.x - conv_blocks) * blockDim.x + threadIdx.x; e < n_e; e += (gridDim.x - conv_blocks) * blockDim.x)
                rc_gate_entry<T>(p + (size_t)(r0 + i) * ld, b_col, a_col, neg_a, dt_bias, beta, lg, r0 + i, e, H, D, per_channel);
        return;
    }
    const int lane = threadIdx.x & 31, it = blockIdx.x * 4 + (threadIdx.x >> 5);
    const int C = 2 * G * D + H * P;
    const int per_warp = 32 / team;                                  // heads a warp takes (team lanes a head)
    const int qk = (2 * G + per_warp - 1) / per_warp;                // items that are q and k heads
    int c[QL];                                                       // this lane's channels (-1: none)
    int head = -1;
    if (it < qk) {
        head = it * per_warp + lane / team;
        if (head >= 2 * G) head = -1;
#pragma unroll
        for (int q = 0; q < QL; q++) {
            const int d = (lane % team + 32 * q) * 4;
            c[q] = head >= 0 && d < D ? head * D + d : -1;
        }
    } else {
#pragma unroll
        for (int q = 0; q < QL; q++) {
            c[q] = 2 * G * D + (it - qk) * 128 * QL + (lane + 32 * q) * 4;
            if (c[q] >= C) c[q] = -1;
        }
    }
    float4 y[RP_ROWS][QL];
#pragma unroll
    for (int q = 0; q < QL; q++) {
        if (c[q] < 0) {
#pragma unroll
            for (int i = 0; i < RP_ROWS; i++) y[i][q] = make_float4(0.f, 0.f, 0.f, 0.f);
            continue;
        }
        float4 win[RP_ROWS + K - 1];
#pragma unroll
        for (int i = 0; i < RP_ROWS + K - 1; i++) {
            const int rr = r0 - (K - 1) + i;
            win[i] = rr >= 0 && rr < n ? rp_load4(p + (size_t)rr * ld + conv_col + c[q]) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        float4 tp[K];
#pragma unroll
        for (int m = 0; m < K; m++)
            tp[m] = make_float4(__ldg(taps + (size_t)c[q] * K + m), __ldg(taps + (size_t)(c[q] + 1) * K + m),
                                __ldg(taps + (size_t)(c[q] + 2) * K + m), __ldg(taps + (size_t)(c[q] + 3) * K + m));
#pragma unroll
        for (int i = 0; i < RP_ROWS; i++) {
            const int r = r0 + i;
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < n) {
                const int seg = row_seg[r], row0 = cu_rows[seg];
                const bool fresh = seg_pos[seg] == 0;
                const float* kp = kept + (size_t)seg_slot[seg] * slot_stride;
#pragma unroll
                for (int m = 0; m < K; m++) {
                    const int rr = r - (K - 1) + m;
                    if (rr >= row0) rp_fma4(acc, tp[m], win[i + m]);
                    else if (!fresh) {
                        const float* k4 = kp + (size_t)(rr - row0 + K - 1) * C + c[q];
                        rp_fma4(acc, tp[m], make_float4(k4[0], k4[1], k4[2], k4[3]));
                    }
                }
            }
            y[i][q] = make_float4(ss_silu(acc.x), ss_silu(acc.y), ss_silu(acc.z), ss_silu(acc.w));
        }
    }
    if (it < qk) {
#pragma unroll
        for (int i = 0; i < RP_ROWS; i++) {
            float ss = 0.f;
#pragma unroll
            for (int q = 0; q < QL; q++) {
                ss = fmaf(y[i][q].x, y[i][q].x, ss); ss = fmaf(y[i][q].y, y[i][q].y, ss);
                ss = fmaf(y[i][q].z, y[i][q].z, ss); ss = fmaf(y[i][q].w, y[i][q].w, ss);
            }
            for (int o = team >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            float scale = 1.0f / sqrtf(ss + RP_UNIT_EPS);
            if (head < G) scale *= q_scale;
#pragma unroll
            for (int q = 0; q < QL; q++) { y[i][q].x *= scale; y[i][q].y *= scale; y[i][q].z *= scale; y[i][q].w *= scale; }
        }
    }
#pragma unroll
    for (int q = 0; q < QL; q++) {
        if (c[q] < 0) continue;
#pragma unroll
        for (int i = 0; i < RP_ROWS; i++)
            if (r0 + i < n) *reinterpret_cast<float4*>(out + (size_t)(r0 + i) * C + c[q]) = y[i][q];
    }
}

// z <- -softplus(-z) / tau in place: the logarithms of the decays sigmoid(z)^(1/tau)
__global__ void log_decay_sigmoid_kernel(float* __restrict__ z, size_t n, float inv_tau) {
    kp_pdl_begin();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        z[i] = rc_log_decay_sigmoid(z[i], inv_tau);
}

// ------------------------------------------------------------------------------------------------ the scan
#define RS_CH 8                  // rows staged at a time
#define RS_COLS 32               // value columns of a block: 8 a warp
#define RS_PARTS 4               // parts the state's rows are cut in: the lanes of a column
#define RS_THREADS 128

// R: state rows a thread keeps (D <= RS_PARTS R).  Lane (part q, column c) owns rows 4 (q + 4 m) + e, m < R / 4, e < 4: the
// four parts read 64 contiguous bytes of a staged vector.  Sums over a column's rows: in a lane by m and e, then the
// lanes by a butterfly.  The read-out is S_new^T q = (g S)^T q + (k . q) u, so that both sums over the old state run
// side by side.
template <typename T, int R, bool DELTA, bool CHAN>
__global__ void __launch_bounds__(RS_THREADS)
recur_scan_kernel(const T* __restrict__ qp, const T* __restrict__ kp, const T* __restrict__ vp, int ldi, const float* __restrict__ lg,
                  const float* __restrict__ beta, float q_scale, float* __restrict__ state, size_t slot_stride,
                  const int* __restrict__ cu_rows, const int* __restrict__ seg_pos, const int* __restrict__ seg_slot,
                  float* __restrict__ out, int ldo, int H, int G, int D, int P, int write_state) {
    kp_pdl_begin();
    constexpr int NP = RS_PARTS * R;
    __shared__ __align__(16) float sq[RS_CH][NP], sk[RS_CH][NP], sg[CHAN ? RS_CH : 1][CHAN ? NP : 4];
    __shared__ float sv[RS_CH][RS_COLS], sdec[RS_CH], sbeta[RS_CH], skq[RS_CH];
    const int head = blockIdx.y, tile = blockIdx.x, seg = blockIdx.z;
    const int grp = head / (H / G);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int col = lane & 7, part = lane >> 3;
    const int jl = warp * 8 + col, j = tile * RS_COLS + jl;
    const bool jok = j < P;
    float* st = state + (size_t)seg_slot[seg] * slot_stride + (size_t)head * D * P;
    const bool fresh = seg_pos[seg] == 0;
    float s[R];
#pragma unroll
    for (int m = 0; m < R / 4; m++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int i = 4 * (part + 4 * m) + e;
            s[4 * m + e] = (!fresh && jok && i < D) ? st[(size_t)i * P + j] : 0.f;
        }
    const int row0 = cu_rows[seg], row1 = cu_rows[seg + 1];
    for (int t0 = row0; t0 < row1; t0 += RS_CH) {
        const int nt = min(RS_CH, row1 - t0);
        __syncthreads();
        for (int t = warp; t < nt; t += RS_THREADS / 32) {
            const size_t row = (size_t)(t0 + t) * ldi;
            float kq = 0.f;
            for (int i = lane; i < NP; i += 32) {
                float qv = 0.f, kv = 0.f, gv = 1.f;
                if (i < D) {
                    qv = to_f32(qp[row + (size_t)grp * D + i]) * q_scale;
                    kv = to_f32(kp[row + (size_t)grp * D + i]);
                    if (CHAN) gv = expf(lg[((size_t)(t0 + t) * H + head) * D + i]);
                }
                sq[t][i] = qv;
                sk[t][i] = kv;
                if (CHAN) sg[t][i] = gv;
                kq = fmaf(qv, kv, kq);
            }
            kq = warp_sum(kq);
            const int jj = tile * RS_COLS + lane;
            sv[t][lane] = jj < P ? to_f32(vp[row + (size_t)head * P + jj]) : 0.f;
            if (lane == 0) {
                skq[t] = kq;
                if (!CHAN) sdec[t] = expf(lg[(size_t)(t0 + t) * H + head]);
                if (DELTA) sbeta[t] = beta[(size_t)(t0 + t) * H + head];
            }
        }
        __syncthreads();
        for (int t = 0; t < nt; t++) {
            const float4* k4 = reinterpret_cast<const float4*>(sk[t]);
            const float4* q4 = reinterpret_cast<const float4*>(sq[t]);
            const float4* g4 = reinterpret_cast<const float4*>(sg[CHAN ? t : 0]);
            const float a = CHAN ? 0.f : sdec[t];
            float ak = 0.f, aq = 0.f;
#pragma unroll
            for (int m = 0; m < R / 4; m++) {
                const float4 kv = k4[part + 4 * m], qv = q4[part + 4 * m];
                const float ke[4] = {kv.x, kv.y, kv.z, kv.w}, qe[4] = {qv.x, qv.y, qv.z, qv.w};
                float ge[4] = {a, a, a, a};
                if (CHAN) {
                    const float4 gv = g4[part + 4 * m];
                    ge[0] = gv.x; ge[1] = gv.y; ge[2] = gv.z; ge[3] = gv.w;
                }
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float x = s[4 * m + e] * ge[e];
                    s[4 * m + e] = x;
                    if (DELTA) ak = fmaf(x, ke[e], ak);
                    aq = fmaf(x, qe[e], aq);
                }
            }
            if (DELTA) {
                ak += __shfl_xor_sync(0xffffffffu, ak, 8);
                ak += __shfl_xor_sync(0xffffffffu, ak, 16);
            }
            aq += __shfl_xor_sync(0xffffffffu, aq, 8);
            aq += __shfl_xor_sync(0xffffffffu, aq, 16);
            const float u = DELTA ? sbeta[t] * (sv[t][jl] - ak) : sv[t][jl];
#pragma unroll
            for (int m = 0; m < R / 4; m++) {
                const float4 kv = k4[part + 4 * m];
                s[4 * m + 0] = fmaf(kv.x, u, s[4 * m + 0]); s[4 * m + 1] = fmaf(kv.y, u, s[4 * m + 1]);
                s[4 * m + 2] = fmaf(kv.z, u, s[4 * m + 2]); s[4 * m + 3] = fmaf(kv.w, u, s[4 * m + 3]);
            }
            if (part == 0 && jok) out[(size_t)(t0 + t) * ldo + (size_t)head * P + j] = fmaf(skq[t], u, aq);
        }
    }
    if (write_state && jok) {
#pragma unroll
        for (int m = 0; m < R / 4; m++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int i = 4 * (part + 4 * m) + e;
                if (i < D) st[(size_t)i * P + j] = s[4 * m + e];
            }
    }
}

// ------------------------------------------------------------------------------------------------ chunked
// For prompt portions in 16-bit mode: a segment in chunks of RC_C rows.  With G_i the sum of the decays' logarithms from
// the chunk's first row up to row i (a number, or one a key channel) and S the state at the chunk's head, the chunk's
// written rows u_i solve the lower triangular system
//   u_i + beta_i sum_{j < i} A_ij u_j = beta_i (v_i - (exp(G_i) k_i)^T S) ,   A_ij = sum_d k_i k_j exp(G_i - G_j) ,
// (in the gated recurrence u = v), and
//   o_i = (exp(G_i) q_i)^T S + sum_{j <= i} B_ij u_j ,                        B_ij = sum_d q_i k_j exp(G_i - G_j) ,
//   S'  = exp(G_last) S + sum_j (exp(G_last - G_j) k_j) u_j^T .
// The system is solved for the right hand sides beta v and beta exp(G) k, so that u = Wv - Wk S; with K' the rows
// exp(G_last - G_j) k_j and Q the rows exp(G_i) q_i everything that depends on S is then one product:
//   S' = M S + N ,   M = diag(exp(G_last)) - K'^T Wk ,   N = K'^T Wv ;        o = (Q - B Wk) S + B Wv .
// Three passes: (0) for all chunks side by side M, N, Q - B Wk, and B Wv into the output rows; (1) a serial pass that walks
// a segment's chunks and leaves every chunk's S in N's place (the gated recurrence: S' = diag(exp(G_last)) S + N, element
// by element); (2) for all chunks side by side the products with S, added to the output rows.
//
// Every exponent is <= 0: where a product of two exponentials stands for exp(G_i - G_j) with factors a channel, its
// reference is a sum that lies between the two; inside eight rows every pair takes its own exponential.
//
// The matrix products run on the tensor cores in tf32 with both operands cut into their upper eleven bits and what those
// leave (three products a pair: what is dropped is about 2^-21 of a term), float32 sums.  What one pass leaves for the
// next lies in the order of the product's register fragments: a tile [16, 8] as 32 lanes of four floats.  As the left
// operand of a product, a result tile's columns 2t and 2t + 1 stand in the places t and t + 4 of the inner index (the
// right operand is read in the same order), so a result is a left operand as it is.
#define RC_C 64
#define RC_LDB 68                // row pitch of the 64 x 64 matrices
#define RC_MAX_D 128
#define RC_MAX_P 256
#define RC_LOG2E 1.4426950408889634f

// 2^x for x <= 0 (the special function unit alone: two units in the last place, below 2^-126 zero)
__device__ __forceinline__ float rc_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void rc_split(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;                       // (by a mask: conversions run at a fraction of its rate)
    lo = __float_as_uint(x - __uint_as_float(hi));               // exact; the product reads its upper bits
}
__device__ __forceinline__ void rc_mma(float* c, const uint32_t* a, const uint32_t* b) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
struct RcA { uint32_t hi[4], lo[4]; };
struct RcB { uint32_t hi[2], lo[2]; };
__device__ __forceinline__ void rc_mma3(float* c, const RcA& a, const RcB& b) {
    rc_mma(c, a.lo, b.hi);
    rc_mma(c, a.hi, b.lo);
    rc_mma(c, a.hi, b.hi);
}
// A tile [16, 8] of an operand stored [row][k]: rows m0 .., columns k0 ..
__device__ __forceinline__ void rc_load_a(RcA& f, const float* s, int ld, int m0, int k0, int g, int t) {
    const float* p = s + (m0 + g) * ld + k0 + t;
    rc_split(p[0], f.hi[0], f.lo[0]);
    rc_split(p[8 * ld], f.hi[1], f.lo[1]);
    rc_split(p[4], f.hi[2], f.lo[2]);
    rc_split(p[8 * ld + 4], f.hi[3], f.lo[3]);
}
// The same of an operand stored [k][row]
__device__ __forceinline__ void rc_load_at(RcA& f, const float* s, int ld, int m0, int k0, int g, int t) {
    const float* p = s + (k0 + t) * ld + m0 + g;
    rc_split(p[0], f.hi[0], f.lo[0]);
    rc_split(p[8], f.hi[1], f.lo[1]);
    rc_split(p[4 * ld], f.hi[2], f.lo[2]);
    rc_split(p[4 * ld + 8], f.hi[3], f.lo[3]);
}
// The same from fragment order (see above)
__device__ __forceinline__ void rc_frag_a(RcA& f, const float4 v) {
    rc_split(v.x, f.hi[0], f.lo[0]);
    rc_split(v.y, f.hi[1], f.lo[1]);
    rc_split(v.z, f.hi[2], f.lo[2]);
    rc_split(v.w, f.hi[3], f.lo[3]);
}
// A tile [8, 8] of a right operand stored [k][col]
__device__ __forceinline__ void rc_load_b(RcB& f, const float* s, int ld, int k0, int n0, int g, int t) {
    const float* p = s + (k0 + t) * ld + n0 + g;
    rc_split(p[0], f.hi[0], f.lo[0]);
    rc_split(p[4 * ld], f.hi[1], f.lo[1]);
}
// The same in the inner order that goes with a left operand in fragment order
__device__ __forceinline__ void rc_load_b2(RcB& f, const float* s, int ld, int k0, int n0, int g, int t) {
    const float* p = s + (k0 + 2 * t) * ld + n0 + g;
    rc_split(p[0], f.hi[0], f.lo[0]);
    rc_split(p[ld], f.hi[1], f.lo[1]);
}
// The same of one stored [col][k]
__device__ __forceinline__ void rc_load_bt(RcB& f, const float* s, int ld, int k0, int n0, int g, int t) {
    const float* p = s + (n0 + g) * ld + k0 + t;
    rc_split(p[0], f.hi[0], f.lo[0]);
    rc_split(p[4], f.hi[1], f.lo[1]);
}

// Sizes: key channels in tiles of 16, value columns in tiles of 8.  What pass 0 leaves of a (chunk, head), in floats: N (then
// S), [D16 / 16][P8 / 8] tiles; Q - B Wk, [4][D16 / 8] tiles; M, [D16 / 16][D16 / 8] tiles, or with the gated recurrence
// exp(G_last) [D16].
struct RcDims { int D16, P8, ld, ldw; };
__host__ __device__ inline RcDims rc_dims(int D, int P, bool delta) {
    RcDims r;
    r.D16 = (D + 15) / 16 * 16;
    r.P8 = (P + 7) / 8 * 8;
    r.ld = (D + 31) / 32 * 32 + 4;                                // (4 beyond a multiple of 32: no bank conflicts by rows)
    r.ldw = (r.P8 + (delta ? r.D16 : 0) + 31) / 32 * 32 + 8;      // (8 beyond: none by columns)
    return r;
}
struct RcRec { size_t n, q, m, size; };
__host__ __device__ inline RcRec rc_record(int D, int P, bool delta) {
    const RcDims s = rc_dims(D, P, delta);
    RcRec r;
    r.n = 0;
    r.q = (size_t)s.D16 * s.P8;
    r.m = r.q + (size_t)RC_C * s.D16;
    r.size = r.m + (delta ? (size_t)s.D16 * s.D16 : s.D16);
    return r;
}
// floats of shared memory of pass 0: K and Q rows, B, exp(G_last), beta, and the sums G and A, whose place W takes later
__host__ inline size_t rc_prepare_floats(int D, int P, bool delta, bool chan) {
    const RcDims s = rc_dims(D, P, delta);
    const size_t ga = (chan ? (size_t)RC_C * s.ld : RC_C) + (delta ? (size_t)RC_C * RC_LDB : 0), w = (size_t)RC_C * s.ldw;
    return 2 * (size_t)RC_C * s.ld + (size_t)RC_C * RC_LDB + s.D16 + RC_C + (ga > w ? ga : w);
}

// Pass 0, one block a (chunk, head).  NTH threads: at least P8 + D16 with the delta rule.
template <typename T, bool DELTA, bool CHAN, int NTH>
__global__ void __launch_bounds__(NTH, 512 / NTH)
recur_chunk_prepare_kernel(const T* __restrict__ qp, const T* __restrict__ kp, const T* __restrict__ vp, int ldi,
                           const float* __restrict__ lg, const float* __restrict__ beta, float q_scale,
                           const int* __restrict__ cu_rows, const int* __restrict__ chunk_seg, const int* __restrict__ chunk_row0,
                           float* __restrict__ rec, float* __restrict__ out, int ldo, int H, int G, int D, int P) {
    kp_pdl_begin();
    constexpr int WARPS = NTH / 32;
    extern __shared__ __align__(16) float rc_sm[];
    const RcDims Z = rc_dims(D, P, DELTA);
    const int ld = Z.ld, Dp = ld - 4;
    float* Ks = rc_sm;                                           // [64][ld]
    float* Qs = Ks + RC_C * ld;                                  // [64][ld]
    float* Bs = Qs + RC_C * ld;                                  // [64][RC_LDB]
    float* el = Bs + RC_C * RC_LDB;                              // [D16]
    float* bt = el + Z.D16;                                      // [64]
    float* Ws = bt + RC_C;                                       // [64][ldw], once the next two are done with
    float* As = Ws;                                              // [64][RC_LDB] (with DELTA)
    float* Gs = As + (DELTA ? RC_C * RC_LDB : 0);                // [64][ld], or [64]: sums of base-2 logarithms
    const int chunk = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane >> 2, t = lane & 3;
    const int grp = head / (H / G);
    const int t0 = chunk_row0[chunk], n = min(RC_C, cu_rows[chunk_seg[chunk] + 1] - t0);
    const RcRec R = rc_record(D, P, DELTA);
    float* dst = rec + ((size_t)chunk * H + head) * R.size;
    // (a warp's rows are fetched together: their loads are all under way before the first is waited for)
    constexpr int ROWS = RC_C / WARPS;
    for (int d = lane; d < Dp; d += 32) {
        float kv[ROWS], qv[ROWS], gv[ROWS];
#pragma unroll
        for (int x = 0; x < ROWS; x++) {
            const int i = warp + x * WARPS;
            const bool ok = i < n && d < D;
            const size_t at = (size_t)(t0 + i) * ldi + (size_t)grp * D + d;
            kv[x] = ok ? to_f32(kp[at]) : 0.f;
            qv[x] = ok ? to_f32(qp[at]) : 0.f;
            gv[x] = CHAN && ok ? lg[((size_t)(t0 + i) * H + head) * D + d] : 0.f;
        }
#pragma unroll
        for (int x = 0; x < ROWS; x++) {
            const int i = warp + x * WARPS;
            Ks[i * ld + d] = kv[x];
            Qs[i * ld + d] = qv[x] * q_scale;
            if (CHAN) Gs[i * ld + d] = gv[x] * RC_LOG2E;
        }
    }
    if (tid < RC_C) {
        bt[tid] = DELTA && tid < n ? beta[(size_t)(t0 + tid) * H + head] : 0.f;
        if (!CHAN) Gs[tid] = tid < n ? lg[(size_t)(t0 + tid) * H + head] * RC_LOG2E : 0.f;
    }
    for (int x = tid; x < RC_C * RC_LDB; x += NTH) Bs[x] = 0.f;  // (what lies above the diagonal is read as part of tiles)
    __syncthreads();
    if (CHAN) {
        for (int d = tid; d < Dp; d += NTH) {
            float acc = 0.f;
#pragma unroll 16
            for (int i = 0; i < RC_C; i++) {
                acc += Gs[i * ld + d];
                Gs[i * ld + d] = acc;
            }
        }
    } else if (warp == 0) {
        const float a = Gs[2 * lane], b = a + Gs[2 * lane + 1];
        float sum = b;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += up;
        }
        float before = __shfl_up_sync(0xffffffffu, sum, 1);
        if (lane == 0) before = 0.f;
        Gs[2 * lane] = before + a;
        Gs[2 * lane + 1] = before + b;
    }
    __syncthreads();
    if (!CHAN) {
        // the ten pieces [16, 16] on and below the diagonal, the warps in turn
        for (int x = warp; x < 10; x += WARPS) {
            const int a = x < 1 ? 0 : (x < 3 ? 1 : (x < 6 ? 2 : 3)), b = x - a * (a + 1) / 2;
            const int m0 = 16 * a, n0 = 16 * b;
            float ca[2][4], cb[2][4];
#pragma unroll
            for (int y = 0; y < 2; y++)
#pragma unroll
                for (int z = 0; z < 4; z++) { ca[y][z] = 0.f; cb[y][z] = 0.f; }
            for (int k0 = 0; k0 < D; k0 += 8) {
                RcA fk, fq;
                if (DELTA) rc_load_a(fk, Ks, ld, m0, k0, g, t);
                rc_load_a(fq, Qs, ld, m0, k0, g, t);
#pragma unroll
                for (int y = 0; y < 2; y++) {
                    RcB fb;
                    rc_load_bt(fb, Ks, ld, k0, n0 + 8 * y, g, t);
                    if (DELTA) rc_mma3(ca[y], fk, fb);
                    rc_mma3(cb[y], fq, fb);
                }
            }
#pragma unroll
            for (int y = 0; y < 2; y++)
#pragma unroll
                for (int z = 0; z < 4; z++) {
                    const int i = m0 + g + (z >> 1) * 8, j = n0 + 8 * y + 2 * t + (z & 1);
                    const float w = j <= i ? rc_exp2(Gs[i] - Gs[j]) : 0.f;
                    if (DELTA) As[i * RC_LDB + j] = j < i ? bt[i] * (w * ca[y][z]) : 0.f;
                    Bs[i * RC_LDB + j] = w * cb[y][z];
                }
        }
    } else {
        // pieces whose rows lie behind their columns: sixteen rows against sixteen earlier ones (six of them), and the upper
        // eight rows of a sixteen against its lower eight (four; their other rows count for nothing).  Both factors by the sum
        // in front of the later rows.
        for (int x = warp; x < 10; x += WARPS) {
            const bool inner = x >= 6;
            const int a = inner ? x - 6 : (x < 1 ? 1 : (x < 3 ? 2 : 3)), b = inner ? a : (x < 1 ? 0 : (x < 3 ? x - 1 : x - 3));
            const int m0 = 16 * a, n0 = 16 * b, ref = inner ? m0 + 7 : m0 - 1;
            const float* Gr = Gs + ref * ld;
            float ca[2][4], cb[2][4];
#pragma unroll
            for (int y = 0; y < 2; y++)
#pragma unroll
                for (int z = 0; z < 4; z++) { ca[y][z] = 0.f; cb[y][z] = 0.f; }
            for (int k0 = 0; k0 < D; k0 += 8) {
                RcA fk, fq;
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int i = m0 + g + (e & 1) * 8, d = k0 + t + (e >> 1) * 4;
                    const float w = i > ref ? rc_exp2(Gs[i * ld + d] - Gr[d]) : 0.f;
                    if (DELTA) rc_split(Ks[i * ld + d] * w, fk.hi[e], fk.lo[e]);
                    rc_split(Qs[i * ld + d] * w, fq.hi[e], fq.lo[e]);
                }
#pragma unroll
                for (int y = 0; y < 2; y++) {
                    if (inner && y) continue;
                    RcB fb;
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const int jj = n0 + y * 8 + g, d = k0 + t + e * 4;
                        rc_split(Ks[jj * ld + d] * rc_exp2(Gr[d] - Gs[jj * ld + d]), fb.hi[e], fb.lo[e]);
                    }
                    if (DELTA) rc_mma3(ca[y], fk, fb);
                    rc_mma3(cb[y], fq, fb);
                }
            }
#pragma unroll
            for (int y = 0; y < 2; y++)
#pragma unroll
                for (int z = 0; z < 4; z++) {
                    const int i = m0 + g + (z >> 1) * 8, jj = n0 + y * 8 + 2 * t + (z & 1);
                    if (i <= ref || (inner && y)) continue;
                    if (DELTA) As[i * RC_LDB + jj] = bt[i] * ca[y][z];
                    Bs[i * RC_LDB + jj] = cb[y][z];
                }
        }
        // pairs inside eight rows: the lanes over the channels
        for (int blk = warp % 8; blk < 8; blk += 8)
            for (int r = warp / 8; r < 8; r += WARPS / 8) {
                const int i = 8 * blk + (WARPS == 8 ? r : (r & 2 ? r ^ 1 : r));
                float ki[RC_MAX_D / 32], qi[RC_MAX_D / 32], gi[RC_MAX_D / 32];
#pragma unroll
                for (int m = 0; m < RC_MAX_D / 32; m++) {
                    const int d = lane + 32 * m;
                    const bool ok = d < Dp;
                    ki[m] = ok && DELTA ? Ks[i * ld + d] : 0.f;
                    qi[m] = ok ? Qs[i * ld + d] : 0.f;
                    gi[m] = ok ? Gs[i * ld + d] : 0.f;
                }
                for (int jj = 8 * blk; jj <= i; jj++) {
                    float sa = 0.f, sb = 0.f;
#pragma unroll
                    for (int m = 0; m < RC_MAX_D / 32; m++) {
                        const int d = lane + 32 * m;
                        if (d < Dp) {
                            const float x = Ks[jj * ld + d] * rc_exp2(gi[m] - Gs[jj * ld + d]);
                            if (DELTA) sa = fmaf(ki[m], x, sa);
                            sb = fmaf(qi[m], x, sb);
                        }
                    }
                    if (DELTA) sa = warp_sum(sa);
                    sb = warp_sum(sb);
                    if (lane == 0) {
                        if (DELTA) As[i * RC_LDB + jj] = jj < i ? bt[i] * sa : 0.f;
                        Bs[i * RC_LDB + jj] = sb;
                    }
                }
            }
    }
    __syncthreads();
    // the right hand sides, one column a thread: beta v, then beta exp(G) k; without DELTA u = v
    const int n_col = Z.P8 + (DELTA ? Z.D16 : 0);
    float w[RC_C];
    if (tid < n_col) {
        const int d = tid - Z.P8;
        if (d < 0) {
            const bool ok = tid < P;
            const T* src = vp + (size_t)t0 * ldi + (size_t)head * P + tid;
#pragma unroll
            for (int i = 0; i < RC_C; i++) w[i] = ok && i < n ? to_f32(src[(size_t)i * ldi]) : 0.f;
            if (DELTA) {
#pragma unroll
                for (int i = 0; i < RC_C; i++) w[i] *= bt[i];
            }
        } else if (d < Dp) {
#pragma unroll
            for (int i = 0; i < RC_C; i++) w[i] = bt[i] * (Ks[i * ld + d] * rc_exp2(CHAN ? Gs[i * ld + d] : Gs[i]));
        }
        if (DELTA) {
#pragma unroll
            for (int i = 1; i < RC_C; i++) {
                float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
                const float4* row = reinterpret_cast<const float4*>(As + i * RC_LDB);
#pragma unroll
                for (int q = 0; q < (i + 3) / 4; q++) {
                    const float4 r4 = row[q];
                    a0 = fmaf(r4.x, w[4 * q], a0);
                    if (4 * q + 1 < i) a1 = fmaf(r4.y, w[4 * q + 1], a1);
                    if (4 * q + 2 < i) a2 = fmaf(r4.z, w[4 * q + 2], a2);
                    if (4 * q + 3 < i) a3 = fmaf(r4.w, w[4 * q + 3], a3);
                }
                w[i] -= (a0 + a1) + (a2 + a3);
            }
        }
    }
    __syncthreads();
    // K and Q rows become exp(G_last - G) k and exp(G) q
    for (int i = warp; i < RC_C; i += WARPS)
        for (int d = lane; d < Dp; d += 32) {
            const float gi = CHAN ? Gs[i * ld + d] : Gs[i], gl = CHAN ? Gs[(RC_C - 1) * ld + d] : Gs[RC_C - 1];
            Ks[i * ld + d] *= rc_exp2(gl - gi);
            Qs[i * ld + d] *= rc_exp2(gi);
        }
    for (int d = tid; d < Z.D16; d += NTH) {
        const float e = d < D ? rc_exp2(CHAN ? Gs[(RC_C - 1) * ld + d] : Gs[RC_C - 1]) : 0.f;
        el[d] = e;
        if (!DELTA) dst[R.m + d] = e;
    }
    __syncthreads();
    if (tid < n_col) {
#pragma unroll
        for (int i = 0; i < RC_C; i++) Ws[i * Z.ldw + tid] = w[i];
    }
    __syncthreads();
    // the products with W: K'^T W (rows: key channels), then B W (rows: the chunk's), four tiles of eight columns an item
    const int mt1 = Z.D16 / 16, tiles = n_col / 8, groups = (tiles + 3) / 4, ks = Z.D16 / 8, nts = Z.P8 / 8;
    for (int x = warp; x < (mt1 + 4) * groups; x += WARPS) {
        const int m = x / groups, n1 = (x - m * groups) * 4;
        const bool first = m < mt1;
        const int m0 = (first ? m : m - mt1) * 16, k_end = first ? RC_C : m0 + 16;
        float acc[4][4];
#pragma unroll
        for (int y = 0; y < 4; y++)
#pragma unroll
            for (int z = 0; z < 4; z++) acc[y][z] = 0.f;
        for (int k0 = 0; k0 < k_end; k0 += 8) {
            RcA fa;
            if (first) rc_load_at(fa, Ks, ld, m0, k0, g, t);
            else rc_load_a(fa, Bs, RC_LDB, m0, k0, g, t);
#pragma unroll
            for (int y = 0; y < 4; y++) {
                RcB fb;
                rc_load_b(fb, Ws, Z.ldw, k0, (n1 + y) * 8, g, t);
                rc_mma3(acc[y], fa, fb);
            }
        }
#pragma unroll
        for (int y = 0; y < 4; y++) {
            const int nt = n1 + y;
            if (nt >= tiles) continue;
            float* c = acc[y];
            if (nt < nts) {
                if (first) {
                    *reinterpret_cast<float4*>(dst + R.n + ((size_t)(m * nts + nt) * 32 + lane) * 4) = make_float4(c[0], c[1], c[2], c[3]);
                } else {
#pragma unroll
                    for (int z = 0; z < 4; z++) {
                        const int i = m0 + g + (z >> 1) * 8, j = nt * 8 + 2 * t + (z & 1);
                        if (i < n && j < P) out[(size_t)(t0 + i) * ldo + (size_t)head * P + j] = c[z];
                    }
                }
            } else if (DELTA) {
                const int k = nt - nts, d = k * 8 + 2 * t;
                if (first) {
                    const int r0 = m0 + g, r1 = r0 + 8;
                    *reinterpret_cast<float4*>(dst + R.m + ((size_t)(m * ks + k) * 32 + lane) * 4) =
                        make_float4((r0 == d ? el[d] : 0.f) - c[0], (r1 == d ? el[d] : 0.f) - c[2],
                                    (r0 == d + 1 ? el[d + 1] : 0.f) - c[1], (r1 == d + 1 ? el[d + 1] : 0.f) - c[3]);
                } else {
                    const float* q0 = Qs + (m0 + g) * ld + d;
                    const float* q1 = q0 + 8 * ld;
                    *reinterpret_cast<float4*>(dst + R.q + ((size_t)((m - mt1) * ks + k) * 32 + lane) * 4) =
                        make_float4(q0[0] - c[0], q1[0] - c[2], q0[1] - c[1], q1[1] - c[3]);
                }
            }
        }
    }
    if (!DELTA) {
        for (int x = warp; x < 4 * ks; x += WARPS) {
            const float* q0 = Qs + (x / ks * 16 + g) * ld + (x % ks) * 8 + 2 * t;
            const float* q1 = q0 + 8 * ld;
            *reinterpret_cast<float4*>(dst + R.q + ((size_t)x * 32 + lane) * 4) = make_float4(q0[0], q1[0], q0[1], q1[1]);
        }
    }
}

// Pass 1 with the delta rule, one block a (16 value columns, head, segment), a warp 16 rows of the state.  In place: N[chunk] <-
// the state at the chunk's head; the segment's slot <- the state behind its last chunk.  The tiles of M come through a ring in
// shared memory, four a stage, STAGES - 1 stages ahead; a lane reads what it has copied itself, so nothing but its own
// copies is waited for.
#define RT_COLS 16
#define RT_STAGES(KS) ((KS) == 16 ? 5 : 6)     // (two blocks an SM at 128 key channels)
#define RT_LD 20                 // (20 % 16 == 4: the right operand's reads, rows 2t and 2t + 1, hit every bank once)
template <int KS>
__global__ void __launch_bounds__(KS * 16, KS == 16 ? 2 : 1)
recur_chunk_states_kernel(float* __restrict__ rec, float* __restrict__ state, size_t slot_stride, const int* __restrict__ seg_pos,
                          const int* __restrict__ seg_slot, const int* __restrict__ seg_chunk0, int H, int D, int P, int write_state) {
    kp_pdl_begin();
    __shared__ __align__(16) float Ss[2][KS * 8 * RT_LD];
    extern __shared__ __align__(16) float rc_sm[];               // [STAGES][4][threads] tiles' float4s
    constexpr int NTH = KS * 16, SPC = KS / 4, STAGES = RT_STAGES(KS);      // (SPC stages a chunk)
    const int head = blockIdx.y, seg = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane >> 2, t = lane & 3;
    const RcDims Z = rc_dims(D, P, true);
    const RcRec R = rc_record(D, P, true);
    const int ks = Z.D16 / 8, nts = Z.P8 / 8, nt0 = blockIdx.x * 2;
    const bool two = nt0 + 1 < nts;
    const size_t step = (size_t)H * R.size;
    const int c0 = seg_chunk0[seg], c1 = seg_chunk0[seg + 1];
    float* base = rec + ((size_t)c0 * H + head) * R.size;
    float* st = state + (size_t)seg_slot[seg] * slot_stride + (size_t)head * D * P;
    const bool fresh = seg_pos[seg] == 0;
    float s[2][4];
#pragma unroll
    for (int y = 0; y < 2; y++)
#pragma unroll
        for (int z = 0; z < 4; z++) {
            const int d = warp * 16 + g + (z >> 1) * 8, j = (nt0 + y) * 8 + 2 * t + (z & 1);
            s[y][z] = !fresh && d < D && j < P ? st[(size_t)d * P + j] : 0.f;
        }
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 nf[2];
    const int total = (c1 - c0) * SPC;
    int put = 0, put_slot = 0, get_slot = 0;                     // the stage to fetch next, its slot, the slot to read next
    auto fetch = [&]() {
        if (put < total) {
            const int c = put / SPC, k0 = put % SPC * 4;
            const float4* src = reinterpret_cast<const float4*>(base + (size_t)c * step + R.m) + (size_t)(warp * ks + k0) * 32 + lane;
#pragma unroll
            for (int i = 0; i < 4; i++)
                if (k0 + i < ks) {
                    const uint32_t a = (uint32_t)__cvta_generic_to_shared(rc_sm + ((put_slot * 4 + i) * NTH + tid) * 4);
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(src + i * 32) : "memory");
                }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        put++;
        put_slot = put_slot + 1 == STAGES ? 0 : put_slot + 1;
    };
    auto n_tile = [&](int c, int y) {
        return c < c1 && (y == 0 || two) ? reinterpret_cast<const float4*>(base + (size_t)(c - c0) * step + R.n)[(size_t)(warp * nts + nt0 + y) * 32 + lane]
                                         : zero;
    };
#pragma unroll
    for (int i = 0; i < STAGES - 1; i++) fetch();
    nf[0] = n_tile(c0, 0);
    nf[1] = n_tile(c0, 1);
    for (int c = c0; c < c1; c++) {
        float* buf = Ss[(c - c0) & 1];
        float4* ns = reinterpret_cast<float4*>(base + (size_t)(c - c0) * step + R.n) + (size_t)(warp * nts + nt0) * 32 + lane;
#pragma unroll
        for (int y = 0; y < 2; y++) {
            float* p = buf + (warp * 16 + g) * RT_LD + y * 8 + 2 * t;
            *reinterpret_cast<float2*>(p) = make_float2(s[y][0], s[y][1]);
            *reinterpret_cast<float2*>(p + 8 * RT_LD) = make_float2(s[y][2], s[y][3]);
            if (y == 0 || two) ns[y * 32] = make_float4(s[y][0], s[y][1], s[y][2], s[y][3]);
        }
        float hi[2][4], lo[2][4];
#pragma unroll
        for (int y = 0; y < 2; y++) {
            hi[y][0] = nf[y].x; hi[y][1] = nf[y].y; hi[y][2] = nf[y].z; hi[y][3] = nf[y].w;
            nf[y] = n_tile(c + 1, y);
#pragma unroll
            for (int z = 0; z < 4; z++) lo[y][z] = 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int part = 0; part < SPC; part++) {
            asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
            const float* tiles = rc_sm + ((size_t)get_slot * 4 * NTH + tid) * 4;
            get_slot = get_slot + 1 == STAGES ? 0 : get_slot + 1;
            float4 m4[4];
#pragma unroll
            for (int i = 0; i < 4; i++) m4[i] = *reinterpret_cast<const float4*>(tiles + i * NTH * 4);
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int k = part * 4 + i;
                if (k >= ks) continue;
                RcA fa;
                rc_frag_a(fa, m4[i]);
#pragma unroll
                for (int y = 0; y < 2; y++) {
                    RcB fb;
                    rc_load_b2(fb, buf, RT_LD, k * 8, y * 8, g, t);
                    rc_mma(lo[y], fa.lo, fb.hi);
                    rc_mma(lo[y], fa.hi, fb.lo);
                    rc_mma(hi[y], fa.hi, fb.hi);
                }
            }
            fetch();                                             // (into the slot read one stage ago)
        }
#pragma unroll
        for (int y = 0; y < 2; y++)
#pragma unroll
            for (int z = 0; z < 4; z++) s[y][z] = hi[y][z] + lo[y][z];
    }
    if (write_state) {
#pragma unroll
        for (int y = 0; y < 2; y++)
#pragma unroll
            for (int z = 0; z < 4; z++) {
                const int d = warp * 16 + g + (z >> 1) * 8, j = (nt0 + y) * 8 + 2 * t + (z & 1);
                if (d < D && j < P) st[(size_t)d * P + j] = s[y][z];
            }
    }
}

// Pass 1 of the gated recurrence, element by element: N[chunk] <- the state at the chunk's head, S' = exp(G_last) S + N.
__global__ void __launch_bounds__(256)
recur_chunk_decay_kernel(float* __restrict__ rec, float* __restrict__ state, size_t slot_stride, const int* __restrict__ seg_pos,
                         const int* __restrict__ seg_slot, const int* __restrict__ seg_chunk0, int H, int D, int P, int write_state) {
    kp_pdl_begin();
    const int head = blockIdx.y, seg = blockIdx.z;
    const int e = blockIdx.x * blockDim.x + threadIdx.x;         // a place in fragment order
    const RcDims Z = rc_dims(D, P, false);
    const RcRec R = rc_record(D, P, false);
    if (e >= Z.D16 * Z.P8) return;
    const int tile = e >> 7, lane = (e >> 2) & 31, z = e & 3, nts = Z.P8 / 8;
    const int d = tile / nts * 16 + (lane >> 2) + (z >> 1) * 8, j = tile % nts * 8 + 2 * (lane & 3) + (z & 1);
    float* st = state + (size_t)seg_slot[seg] * slot_stride + ((size_t)head * D + d) * P + j;
    const bool real = d < D && j < P;
    float S = real && seg_pos[seg] != 0 ? *st : 0.f;
    const size_t step = (size_t)H * R.size;
    const int c_end = seg_chunk0[seg + 1];
    for (int c0 = seg_chunk0[seg]; c0 < c_end; c0 += 8) {
        float* p = rec + ((size_t)c0 * H + head) * R.size;
        float u[8], w[8];
#pragma unroll
        for (int k = 0; k < 8; k++)
            if (c0 + k < c_end) {
                u[k] = p[k * step + R.n + e];
                w[k] = p[k * step + R.m + d];
            }
#pragma unroll
        for (int k = 0; k < 8; k++)
            if (c0 + k < c_end) {
                p[k * step + R.n + e] = S;
                S = fmaf(w[k], S, u[k]);
            }
    }
    if (write_state && real) *st = S;
}

// Pass 2, one block a (64 value columns, chunk, head): out += (Q - B Wk) S.
#define RO_COLS 64
#define RO_LD 68                 // (68 % 16 == 4)
#define RO_THREADS 256
__global__ void __launch_bounds__(RO_THREADS)
recur_chunk_out_kernel(const float* __restrict__ rec, const int* __restrict__ cu_rows, const int* __restrict__ chunk_seg,
                       const int* __restrict__ chunk_row0, float* __restrict__ out, int ldo, int H, int D, int P, int delta) {
    kp_pdl_begin();
    __shared__ __align__(16) float Ss[RC_MAX_D * RO_LD];
    const int chunk = blockIdx.y, head = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int g = lane >> 2, t = lane & 3;
    const int t0 = chunk_row0[chunk], n = min(RC_C, cu_rows[chunk_seg[chunk] + 1] - t0);
    const RcDims Z = rc_dims(D, P, delta != 0);
    const RcRec R = rc_record(D, P, delta != 0);
    const float* src = rec + ((size_t)chunk * H + head) * R.size;
    const int ks = Z.D16 / 8, nts = Z.P8 / 8, nt0 = blockIdx.x * (RO_COLS / 8), tiles = min(RO_COLS / 8, nts - nt0);
    for (int x = warp; x < (Z.D16 / 16) * (RO_COLS / 8); x += RO_THREADS / 32) {
        const int m = x / (RO_COLS / 8), y = x % (RO_COLS / 8);
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (y < tiles) v = __ldg(reinterpret_cast<const float4*>(src + R.n) + (size_t)(m * nts + nt0 + y) * 32 + lane);
        float* p = Ss + (m * 16 + g) * RO_LD + y * 8 + 2 * t;
        *reinterpret_cast<float2*>(p) = make_float2(v.x, v.y);
        *reinterpret_cast<float2*>(p + 8 * RO_LD) = make_float2(v.z, v.w);
    }
    __syncthreads();
    const int m = warp & 3, n0 = (warp >> 2) * 4;                // 16 rows, four tiles of eight columns
    if (m * 16 >= n || n0 >= tiles) return;
    float acc[4][4];
#pragma unroll
    for (int y = 0; y < 4; y++)
#pragma unroll
        for (int z = 0; z < 4; z++) acc[y][z] = 0.f;
    const float4* qf = reinterpret_cast<const float4*>(src + R.q) + (size_t)m * ks * 32 + lane;
#pragma unroll 4
    for (int k = 0; k < ks; k++) {
        RcA fa;
        rc_frag_a(fa, __ldg(qf + (size_t)k * 32));
#pragma unroll
        for (int y = 0; y < 4; y++) {
            RcB fb;
            rc_load_b2(fb, Ss, RO_LD, k * 8, (n0 + y) * 8, g, t);
            rc_mma3(acc[y], fa, fb);
        }
    }
#pragma unroll
    for (int y = 0; y < 4; y++)
#pragma unroll
        for (int z = 0; z < 4; z++) {
            const int i = m * 16 + g + (z >> 1) * 8, j = (nt0 + n0 + y) * 8 + 2 * t + (z & 1);
            if (i < n && j < P) out[(size_t)(t0 + i) * ldo + (size_t)head * P + j] += acc[y][z];
        }
}

extern "C" {

// Convolutions, unit norms, step sizes and decays in front of a delta recurrence: see delta_prep_kernel.  per_channel: lg
// holds the decays' projections [n, H D] and is changed in place; else they are columns a_col .. of p and lg [n, H] is
// written.  taps [C][K]; neg_a [H]: -exp(A_log); dt_bias [H D] or [H].  kept: a slot's last K - 1 inputs at `kept + slot *
// slot_stride`; renewed unless keep == 0 (single_rows: by the same launch, else by a second one).
int kp_delta_prep(const void* p, int ld, int conv_col, int b_col, int a_col, const float* taps, const float* neg_a,
                  const float* dt_bias, float* kept, long long slot_stride, const int* row_seg, const int* cu_rows, const int* seg_pos,
                  const int* seg_slot, float* out, float* beta, float* lg, int n, int n_seg, int H, int G, int D, int P, int K,
                  float q_scale, int per_channel, int single_rows, int keep, int dtype, void* stream) {
    if (n <= 0) return 0;
    if (H < 1 || G < 1 || H % G || D < 1 || P < 1) return KP_ERR_BAD_ARG;
    if (D > 256 || K < 1 || K > SS_MAX_TAPS || n > 65535 || n_seg > 65535) return KP_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const int C = 2 * G * D + H * P, n_e = H + (per_channel ? H * D : H);
    const int esz = dtype == KP_DTYPE_F32 ? 4 : 2;
    const bool vec = !single_rows && K <= 4 && n >= 2 * RP_ROWS && D % 4 == 0 && (H * P) % 4 == 0 && ld % 4 == 0 && conv_col % 4 == 0 &&
                     (uintptr_t)p % (4 * esz) == 0 && (uintptr_t)out % 16 == 0;
    if (vec) {
        const int quads = D / 4, team = (quads & (quads - 1)) == 0 && quads <= 32 ? quads : 32;
        const int ql = D > 128 ? 2 : 1, per_warp = 32 / team;
        const int items = (2 * G + per_warp - 1) / per_warp + (H * P + 128 * ql - 1) / (128 * ql);
        const int conv_blocks = (items + 3) / 4;
        int gate_blocks = (n_e + 127) / 128;
        if (gate_blocks > 32) gate_blocks = 32;
        const dim3 grid(conv_blocks + gate_blocks, (n + RP_ROWS - 1) / RP_ROWS);
#define RP_LAUNCH(KK, QQ)                                                                                                    \
        KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(delta_prep_vec_kernel<T, KK, QQ>, grid, dim3(128), 0, s, (const T*)p, ld, conv_col, b_col, \
                                                   a_col, taps, neg_a, dt_bias, (const float*)kept, (size_t)slot_stride, row_seg, cu_rows,   \
                                                   seg_pos, seg_slot, out, beta, lg, n, H, G, D, P, q_scale, per_channel, conv_blocks, team)))
#define RP_LAUNCH_K(QQ)                                                                                                      \
        do { if (K == 1) RP_LAUNCH(1, QQ); else if (K == 2) RP_LAUNCH(2, QQ); else if (K == 3) RP_LAUNCH(3, QQ); else RP_LAUNCH(4, QQ); } while (0)
        if (ql == 1) RP_LAUNCH_K(1);
        else RP_LAUNCH_K(2);
#undef RP_LAUNCH_K
#undef RP_LAUNCH
    } else {
        const int items = 2 * G + (H * P + 127) / 128 + (n_e + 127) / 128;
        KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(delta_prep_kernel<T>, dim3((items + 3) / 4, n), dim3(128), 0, s, (const T*)p, ld, conv_col,
                                                   b_col, a_col, taps, neg_a, dt_bias, kept, (size_t)slot_stride, row_seg, cu_rows, seg_pos,
                                                   seg_slot, out, beta, lg, H, G, D, P, K, q_scale, per_channel, single_rows && keep)));
    }
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) return (int)e;
    if (keep && !single_rows && K > 1) {
        KP_DISPATCH_DTYPE(dtype, T, (kp_launch_pdl(ssm_conv_keep_kernel<T>, dim3((C + 127) / 128, n_seg), dim3(128), 0, s, (const T*)p, ld,
                                                   conv_col, kept, (size_t)slot_stride, cu_rows, seg_pos, seg_slot, C, K)));
    }
    return kp_launch_status();
}

int kp_log_decay_sigmoid(float* z, long long n, float inv_tau, void* stream) {
    if (n <= 0) return 0;
    long long blocks = (n + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    kp_launch_pdl(log_decay_sigmoid_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, z, (size_t)n, inv_tau);
    return kp_launch_status();
}

// q, k (G heads of D) and v (H heads of P): rows of pitch ldi, in float32 or the storage type (dtype).  lg: [n, H] or, with
// per_channel, [n, H D] float32; beta: [n, H], or null for the gated recurrence.  state: a slot's [H][D][P] float32 at
// `state + slot * slot_stride`.  out: [n, ldo] float32, heads side by side.
int kp_recur_scan(const void* q, const void* k, const void* v, int ldi, const float* lg, const float* beta, float q_scale, float* state,
                  long long slot_stride, const int* cu_rows, const int* seg_pos, const int* seg_slot, float* out, int ldo, int n_seg,
                  int H, int G, int D, int P, int per_channel, int write_state, int dtype, void* stream) {
    if (n_seg <= 0) return 0;
    if (H < 1 || G < 1 || H % G || D < 1 || P < 1) return KP_ERR_BAD_ARG;
    if (D > 256 || H > 65535 || n_seg > 65535) return KP_ERR_UNSUPPORTED;
    const dim3 grid((P + RS_COLS - 1) / RS_COLS, H, n_seg), block(RS_THREADS);
    cudaStream_t s = (cudaStream_t)stream;
#define RS_LAUNCH(T, R, DL, CH)                                                                                              \
    kp_launch_pdl(recur_scan_kernel<T, R, DL, CH>, grid, block, 0, s, (const T*)q, (const T*)k, (const T*)v, ldi, lg, beta, q_scale, state,  \
                  (size_t)slot_stride, cu_rows, seg_pos, seg_slot, out, ldo, H, G, D, P, write_state)
#define RS_LAUNCH_R(T, DL, CH)                                                                                               \
    do {                                                                                                                     \
        if (D <= 32) RS_LAUNCH(T, 8, DL, CH);                                                                                \
        else if (D <= 64) RS_LAUNCH(T, 16, DL, CH);                                                                          \
        else if (D <= 128) RS_LAUNCH(T, 32, DL, CH);                                                                         \
        else RS_LAUNCH(T, 64, DL, CH);                                                                                       \
    } while (0)
    // (the rows a thread keeps depend on the state's size only, so a row's sums have the same order in every launch)
    if (beta) {
        if (dtype != KP_DTYPE_F32) return KP_ERR_UNSUPPORTED;          // (what delta_prep leaves)
        if (per_channel) RS_LAUNCH_R(float, true, true);
        else RS_LAUNCH_R(float, true, false);
    } else {
        if (!per_channel) return KP_ERR_UNSUPPORTED;
        KP_DISPATCH_DTYPE(dtype, T, RS_LAUNCH_R(T, false, true));
    }
#undef RS_LAUNCH_R
#undef RS_LAUNCH
    return kp_launch_status();
}

int kp_recur_chunk_rows() { return RC_C; }
int kp_recur_chunks_ok(int D, int P) { return D >= 1 && P >= 1 && D <= RC_MAX_D && P <= RC_MAX_P; }
// floats of scratch that kp_recur_chunks wants: the records of pass 0
long long kp_recur_chunks_scratch(int n_chunks, int H, int D, int P, int delta) {
    return (long long)n_chunks * H * (long long)rc_record(D, P, delta != 0).size;
}

// The chunked form: the arguments of kp_recur_scan and the list of chunks (chunk_seg, chunk_row0 [n_chunks]: every chunk's
// segment, numbered among the n_seg segments given here, and first row; seg_chunk0 [n_seg + 1]: the first chunk of every
// segment).  scratch: kp_recur_chunks_scratch floats, 16-byte aligned.  KP_ERR_UNSUPPORTED for sizes that
// kp_recur_chunks_ok does not take.
int kp_recur_chunks(const void* q, const void* k, const void* v, int ldi, const float* lg, const float* beta, float q_scale, float* state,
                    long long slot_stride, const int* cu_rows, const int* seg_pos, const int* seg_slot, const int* chunk_seg,
                    const int* chunk_row0, const int* seg_chunk0, int n_chunks, float* scratch, float* out, int ldo, int n_seg, int H,
                    int G, int D, int P, int per_channel, int write_state, int dtype, void* stream) {
    if (n_seg <= 0 || n_chunks <= 0) return 0;
    if (H < 1 || G < 1 || H % G || D < 1 || P < 1 || (uintptr_t)scratch % 16) return KP_ERR_BAD_ARG;
    if (!kp_recur_chunks_ok(D, P) || H > 65535 || n_seg > 65535 || n_chunks > 65535) return KP_ERR_UNSUPPORTED;
    const bool delta = beta != nullptr;
    const RcDims Z = rc_dims(D, P, delta);
    const size_t sm0 = rc_prepare_floats(D, P, delta, per_channel != 0) * sizeof(float);
    // (256 threads, two blocks an SM, where a column a thread and the shared memory allow it)
    const bool small = Z.P8 + (delta ? Z.D16 : 0) <= 256 && sm0 <= 112 * 1024;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
#define RC_PREPARE_N(T, DL, CH, NTH)                                                                                         \
    do {                                                                                                                     \
        if ((e = cudaFuncSetAttribute(recur_chunk_prepare_kernel<T, DL, CH, NTH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm0)) != cudaSuccess) \
            return (int)e;                                                                                                   \
        kp_launch_pdl(recur_chunk_prepare_kernel<T, DL, CH, NTH>, dim3(n_chunks, H), dim3(NTH), sm0, s, (const T*)q, (const T*)k, (const T*)v, \
                      ldi, lg, beta, q_scale, cu_rows, chunk_seg, chunk_row0, scratch, out, ldo, H, G, D, P);                \
    } while (0)
#define RC_PREPARE(T, DL, CH) do { if (small) RC_PREPARE_N(T, DL, CH, 256); else RC_PREPARE_N(T, DL, CH, 512); } while (0)
    if (delta) {
        if (dtype != KP_DTYPE_F32) return KP_ERR_UNSUPPORTED;          // (what delta_prep leaves)
        if (per_channel) RC_PREPARE(float, true, true);
        else RC_PREPARE(float, true, false);
    } else {
        if (!per_channel) return KP_ERR_UNSUPPORTED;
        KP_DISPATCH_DTYPE(dtype, T, RC_PREPARE(T, false, true));
    }
#undef RC_PREPARE
#undef RC_PREPARE_N
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
    if (delta) {
        const dim3 grid((Z.P8 + RT_COLS - 1) / RT_COLS, H, n_seg), block(Z.D16 * 2);
        // (a ring as wide as the kernel's largest block: its pitch does not depend on the block that is launched)
#define RC_STATES(KS)                                                                                                        \
        do {                                                                                                                 \
            const size_t ring = (size_t)RT_STAGES(KS) * 4 * (KS * 16) * 16;                                                      \
            if ((e = cudaFuncSetAttribute(recur_chunk_states_kernel<KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ring)) != cudaSuccess) \
                return (int)e;                                                                                               \
            kp_launch_pdl(recur_chunk_states_kernel<KS>, grid, block, ring, s, scratch, state, (size_t)slot_stride, seg_pos, seg_slot, \
                          seg_chunk0, H, D, P, write_state);                                                                 \
        } while (0)
        if (D <= 32) RC_STATES(4);
        else if (D <= 64) RC_STATES(8);
        else RC_STATES(16);
#undef RC_STATES
    } else {
        kp_launch_pdl(recur_chunk_decay_kernel, dim3((Z.D16 * Z.P8 + 255) / 256, H, n_seg), dim3(256), 0, s, scratch, state, (size_t)slot_stride,
                      seg_pos, seg_slot, seg_chunk0, H, D, P, write_state);
    }
    if ((e = cudaGetLastError()) != cudaSuccess) return (int)e;
    kp_launch_pdl(recur_chunk_out_kernel, dim3((Z.P8 + RO_COLS - 1) / RO_COLS, n_chunks, H), dim3(RO_THREADS), 0, s, (const float*)scratch, cu_rows,
                  chunk_seg, chunk_row0, out, ldo, H, D, P, (int)delta);
    return kp_launch_status();
}

}  // extern "C"
