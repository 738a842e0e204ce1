// The gated delta rule with one decay per head and token, in chunks of 64 tokens on the tensor cores:
//
//   S <- e^{a_i} S;   u_i = beta_i (v_i - S^T k_i);   S <- S + k_i u_i^T;   o_i = S^T q_i
//
// With L_i the sum of a over a chunk's tokens up to i and S the state in front of the chunk, what the tokens write solves a unit lower
// triangular system,
//
//   (I + A) U = diag(beta) V - diag(beta e^L) K S,      A_ij = beta_i e^{L_i - L_j} (k_i . k_j) for j < i,
//
// so with T = (I + A)^{-1}:  U = U0 - W S,  U0 = T diag(beta) V,  W = T diag(beta e^L) K, and behind the chunk e^{L_n} S + sum_j
// e^{L_n - L_j} k_j u_j^T.  Kernels of a step:
//
//   steps    per token: a and beta per head, the factors that make q and k unit vectors (q's times d^-1/2), float32
//   solve    per (chunk, head): A on the tensor cores, T by substitution in float32, W and U0
//   state    per (request, head, 16 value columns): the chunks in order with the state in registers; leaves U and, in front of every
//            chunk, the state
//   (out)    decay_chunks.cu: o, norm per head, weight, gate, all chunks at once
//
// k and q are bfloat16 operands as the convolutions leave them; their unit factors multiply scores and columns in float32.  T, W, U and
// the states are float32 and enter a product as two bfloat16 terms.
#include "decay_chunks.cuh"
#include <math.h>

#define DL_NC 16                 // value columns of a CTA of the state kernel
#define DL_LDS (DL_NC + 8)

// a warp a head row: queries, then keys; then the value heads' numbers
__global__ void __launch_bounds__(128)
delta_steps_kernel(const __nv_bfloat16 *__restrict__ act, long long ld_act, const float *__restrict__ p, int S, size_t slice_stride, int ld, int col_beta,
                   int col_a, const float *__restrict__ A_log, const float *__restrict__ dt_bias, float *__restrict__ q_scale, float *__restrict__ k_scale,
                   float *__restrict__ beta, float *__restrict__ log_decay, int H, int G, int d) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float mul = 1.0f / sqrtf((float)d);
    for (int r = warp; r < 2 * G; r += 4) {
        const __nv_bfloat16 *x = act + (size_t)t * ld_act + (size_t)r * d;
        float ss = 0.f;
        for (int i = 2 * lane; i < d; i += 64) {
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162 *>(x + i);
            const float a = __bfloat162float(v.x), b = __bfloat162float(v.y);
            ss = fmaf(a, a, fmaf(b, b, ss));
        }
        ss = warp_sum(ss);
        if (lane == 0) {
            const float inv = 1.0f / sqrtf(ss + 1e-6f);
            if (r < G) q_scale[(size_t)t * G + r] = inv * mul;
            else k_scale[(size_t)t * G + r - G] = inv;
        }
    }
    for (int h = threadIdx.x; h < H; h += 128) {
        const float z = sum_slices(p, S, slice_stride, (size_t)t * ld + col_beta + h);
        const float a = sum_slices(p, S, slice_stride, (size_t)t * ld + col_a + h) + dt_bias[h];
        beta[(size_t)t * H + h] = 1.0f / (1.0f + expf(-z));
        log_decay[(size_t)t * H + h] = -expf(A_log[h]) * (a > 20.f ? a : log1pf(expf(a)));
    }
}

struct DeltaChunkParams {
    const __nv_bfloat16 *act;            // rows [q: G d | k: G d | v: H dv]
    long long ld_act;
    int G;
    const float *k_scale, *beta, *log_decay;
    const int *cu_seqlens, *slots, *tile_seq, *tile_row0, *first_tile;
    __nv_bfloat16 *w_hi, *w_lo;          // [tiles, H, 64, d]
    float *u0;                           // [tiles, H, 64, dv]
    float *factors;                      // [tiles, H, 68]: e^{L_n - L_j} times k's unit factor for the 64 tokens, then e^{L_n}
    float *state;
    long long state_stride, state_off;
    __nv_bfloat16 *before;               // [tiles, H, 2, d, dv]
    __nv_bfloat16 *u_hi, *u_lo;          // [T, H dv]
    int H, d, dv;
};

template <int D>
__global__ void __launch_bounds__(128)
delta_chunk_solve_kernel(const DeltaChunkParams p) {
    constexpr int LDA = 68;
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t dl_raw[];
    float *A = reinterpret_cast<float *>(dl_raw);                              // [64][LDA]
    __nv_bfloat16 *Ks = reinterpret_cast<__nv_bfloat16 *>(A + DC_C * LDA), *Vs = Ks + DC_C * (D + 8);
    __nv_bfloat16 *Wh = Vs + DC_C * DC_LDN, *Wl = Wh + DC_C * DC_LDN, *Uh = Wl + DC_C * DC_LDN, *Ul = Uh + DC_C * DC_LDN;      // T's columns times what W and U0 take
    __shared__ float L[DC_C], kf[DC_C], bt[DC_C];
    const int tile = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = p.tile_seq[tile], row0 = p.tile_row0[tile], tb = p.cu_seqlens[seq], n = min(DC_C, p.cu_seqlens[seq + 1] - tb - row0);
    const int d = p.d, dv = p.dv, G = p.G, hk = h / (p.H / G);
    const size_t t0 = (size_t)tb + row0, th = (size_t)tile * p.H + h;
    const __nv_bfloat16 *k_src = p.act + t0 * p.ld_act + (size_t)(G + hk) * d, *v_src = p.act + t0 * p.ld_act + 2 * (size_t)G * d + (size_t)h * dv;
    auto load_v = [&](int n0) {
        for (int idx = tid; idx < DC_C * (DC_N / 8); idx += 128) {
            const int r = idx / (DC_N / 8), c = idx % (DC_N / 8) * 8;
            const bool ok = r < n && n0 + c < dv;
            dc_cp16(Vs + r * DC_LDN + c, v_src + (ok ? (size_t)r * p.ld_act + n0 + c : 0), ok);
        }
        dc_commit();
    };
    dc_load_rows<D>(Ks, k_src, p.ld_act, n, d, tid);
    dc_commit();
    load_v(0);
    dc_running_sums(L, p.log_decay + t0 * p.H + h, p.H, n, tid);
    if (tid >= 64) {
        const int j = tid - 64;
        kf[j] = j < n ? p.k_scale[(t0 + j) * G + hk] : 0.f;
        bt[j] = j < n ? p.beta[(t0 + j) * p.H + h] : 0.f;
    }
    dc_wait<1>();
    __syncthreads();
    if (tid < DC_C) p.factors[th * 68 + tid] = __expf(L[DC_C - 1] - L[tid]) * kf[tid];
    if (tid == DC_C) p.factors[th * 68 + DC_C] = expf(L[DC_C - 1]);
    const int g = lane >> 2, tq = lane & 3;
    const int a_row = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, a_k = (lane >> 4) * 8;
    const int b_row = (lane & 7) + (lane >> 4) * 8, b_k = ((lane >> 3) & 1) * 8;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    {
        float s[DC_C / 8][4];
#pragma unroll
        for (int j = 0; j < DC_C / 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[j][c] = 0.f;
        for (int kk = 0; kk < (d + 15) / 16; ++kk) {
            uint32_t a[4];
            ldmatrix_x4(dc_smem(Ks + a_row * (D + 8) + kk * 16 + a_k), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int jp = 0; jp < DC_C / 16; ++jp) {
                if (jp > warp) continue;
                uint32_t b00, b01, b10, b11;
                ldmatrix_x4(dc_smem(Ks + (jp * 16 + b_row) * (D + 8) + kk * 16 + b_k), b00, b01, b10, b11);
                mma_bf16(s[2 * jp], a, b00, b01);
                mma_bf16(s[2 * jp + 1], a, b10, b11);
            }
        }
#pragma unroll
        for (int jt = 0; jt < DC_C / 8; ++jt)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = warp * 16 + g + 8 * hf, j = jt * 8 + 2 * tq;
                const float f = bt[i] * kf[i];
                const float x0 = i > j ? s[jt][2 * hf] * (f * kf[j] * __expf(L[i] - L[j])) : 0.f;
                const float x1 = i > j + 1 ? s[jt][2 * hf + 1] * (f * kf[j + 1] * __expf(L[i] - L[j + 1])) : 0.f;
                *reinterpret_cast<float2 *>(A + i * LDA + j) = make_float2(x0, x1);
            }
    }
    __syncthreads();
    if (tid < DC_C) {                                 // a thread a column of T: x_j = 1, x_i = -sum_{m < i} A_im x_m
        float x[DC_C];
#pragma unroll
        for (int i = 0; i < DC_C; ++i) {
            float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
            for (int m = 0; m + 3 < i; m += 4) {
                const float4 a = *reinterpret_cast<const float4 *>(A + i * LDA + m);
                s0 = fmaf(a.x, x[m], s0);
                s1 = fmaf(a.y, x[m + 1], s1);
                s2 = fmaf(a.z, x[m + 2], s2);
                s3 = fmaf(a.w, x[m + 3], s3);
            }
#pragma unroll
            for (int m = i / 4 * 4; m < i; ++m) s0 = fmaf(A[i * LDA + m], x[m], s0);
            x[i] = i < tid ? 0.f : (i == tid ? 1.f : -((s0 + s1) + (s2 + s3)));
        }
        const float fu = bt[tid], fw = fu * kf[tid] * __expf(L[tid]);
#pragma unroll
        for (int i = 0; i < DC_C; ++i) {
            dc_split(x[i] * fw, Wh[i * DC_LDN + tid], Wl[i * DC_LDN + tid]);
            dc_split(x[i] * fu, Uh[i * DC_LDN + tid], Ul[i * DC_LDN + tid]);
        }
    }
    dc_wait<0>();
    __syncthreads();
    // W = T' K: this warp's 16 rows, 64 columns at a time
    for (int n0 = 0; n0 < d; n0 += 64) {
        float acc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[j][c] = 0.f;
        for (int kk = 0; kk <= warp; ++kk) {          // T is lower triangular
            uint32_t a[4], al[4];
            ldmatrix_x4(dc_smem(Wh + a_row * DC_LDN + kk * 16 + a_k), a[0], a[1], a[2], a[3]);
            ldmatrix_x4(dc_smem(Wl + a_row * DC_LDN + kk * 16 + a_k), al[0], al[1], al[2], al[3]);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                if (n0 + np * 16 >= D) continue;
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(dc_smem(Ks + (kk * 16 + v_row) * (D + 8) + n0 + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(acc[2 * np], a, b0, b1);
                mma_bf16(acc[2 * np + 1], a, b2, b3);
                mma_bf16(acc[2 * np], al, b0, b1);
                mma_bf16(acc[2 * np + 1], al, b2, b3);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int col = n0 + j * 8 + 2 * tq;
            if (col >= d) continue;
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const size_t o = (th * DC_C + warp * 16 + g + 8 * hf) * d + col;
                uint32_t hi, lo;
                dc_split2(acc[j][2 * hf], acc[j][2 * hf + 1], hi, lo);
                *reinterpret_cast<uint32_t *>(p.w_hi + o) = hi;
                *reinterpret_cast<uint32_t *>(p.w_lo + o) = lo;
            }
        }
    }
    for (int n0 = 0; n0 < dv; n0 += DC_N) {
        if (n0 > 0) {
            __syncthreads();
            load_v(n0);
            dc_wait<0>();
            __syncthreads();
        }
        float acc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[j][c] = 0.f;
        for (int kk = 0; kk <= warp; ++kk) {
            uint32_t a[4], al[4];
            ldmatrix_x4(dc_smem(Uh + a_row * DC_LDN + kk * 16 + a_k), a[0], a[1], a[2], a[3]);
            ldmatrix_x4(dc_smem(Ul + a_row * DC_LDN + kk * 16 + a_k), al[0], al[1], al[2], al[3]);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(dc_smem(Vs + (kk * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(acc[2 * np], a, b0, b1);
                mma_bf16(acc[2 * np + 1], a, b2, b3);
                mma_bf16(acc[2 * np], al, b0, b1);
                mma_bf16(acc[2 * np + 1], al, b2, b3);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int col = n0 + j * 8 + 2 * tq;
            if (col >= dv) continue;
#pragma unroll
            for (int hf = 0; hf < 2; ++hf)
                *reinterpret_cast<float2 *>(p.u0 + (th * DC_C + warp * 16 + g + 8 * hf) * dv + col) = make_float2(acc[j][2 * hf], acc[j][2 * hf + 1]);
        }
    }
}

// The chunks of a request in order, 16 value columns of a head.  The state's rows sit in the warps' accumulators; as the operand of the
// next chunk's product it goes through shared memory in two terms.
template <int D>
__global__ void __launch_bounds__(128)
delta_chunk_state_kernel(const DeltaChunkParams p) {
    constexpr int MT = D >= 64 ? D / 64 : 1;          // 16-row tiles of the state a warp keeps
    constexpr int STAGE = 3 * DC_C * (D + 8);
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t dl_raw[];
    __nv_bfloat16 *stages = reinterpret_cast<__nv_bfloat16 *>(dl_raw);         // 2 x { W_hi, W_lo, K }
    __nv_bfloat16 *Sh = stages + 2 * STAGE, *Sl = Sh + D * DL_LDS, *Uh = Sl + D * DL_LDS, *Ul = Uh + DC_C * DL_LDS;
    const int n0 = blockIdx.x * DL_NC, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int lo = p.first_tile[seq], hi = p.first_tile[seq + 1];
    if (lo == hi) return;
    const int d = p.d, dv = p.dv, G = p.G, hk = h / (p.H / G), tb = p.cu_seqlens[seq], te = p.cu_seqlens[seq + 1];
    const int g = lane >> 2, tq = lane & 3;
    const int a_row = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, a_kk = (lane >> 4) * 8;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    const int t_k = (lane & 7) + (lane >> 4) * 8, t_m = ((lane >> 3) & 1) * 8;
    float *st = p.state + (size_t)p.slots[seq] * p.state_stride + p.state_off + (size_t)h * d * dv;
    float S[MT][2][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int i = (warp + 4 * m) * 16 + g + 8 * (c >> 1), col = n0 + j * 8 + 2 * tq + (c & 1);
                S[m][j][c] = i < d && col < dv ? st[(size_t)i * dv + col] : 0.f;
            }
    auto issue = [&](int tile, int stage) {
        __nv_bfloat16 *w = stages + stage * STAGE;
        const size_t th = (size_t)tile * p.H + h;
        const int row0 = (tile - lo) * DC_C, n = min(DC_C, te - tb - row0);
        dc_load_rows<D>(w, p.w_hi + th * DC_C * d, d, DC_C, d, tid);
        dc_load_rows<D>(w + DC_C * (D + 8), p.w_lo + th * DC_C * d, d, DC_C, d, tid);
        dc_load_rows<D>(w + 2 * DC_C * (D + 8), p.act + ((size_t)tb + row0) * p.ld_act + (size_t)(G + hk) * d, p.ld_act, n, d, tid);
    };
    issue(lo, 0);
    dc_commit();
    for (int tile = lo; tile < hi; ++tile) {
        const int stage = (tile - lo) & 1, row0 = (tile - lo) * DC_C, n = min(DC_C, te - tb - row0);
        const size_t th = (size_t)tile * p.H + h;
        const __nv_bfloat16 *W1 = stages + stage * STAGE, *W2 = W1 + DC_C * (D + 8), *Ks = W2 + DC_C * (D + 8);
        if (tile + 1 < hi) issue(tile + 1, stage ^ 1);
        dc_commit();
        // what the products' results meet, on its way meanwhile
        float2 u0[2][2];
        float kf[2];
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const int i = warp * 16 + g + 8 * hf;
            kf[hf] = p.factors[th * 68 + i];
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int col = n0 + j * 8 + 2 * tq;
                u0[hf][j] = col < dv ? *reinterpret_cast<const float2 *>(p.u0 + (th * DC_C + i) * dv + col) : make_float2(0.f, 0.f);
            }
        }
        const float total = p.factors[th * 68 + DC_C];
        __nv_bfloat16 *before = p.before + th * 2 * d * dv;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const int i = (warp + 4 * m) * 16 + g + 8 * hf, c = j * 8 + 2 * tq;
                    if (i >= D) continue;
                    uint32_t x, y;
                    dc_split2(S[m][j][2 * hf], S[m][j][2 * hf + 1], x, y);
                    *reinterpret_cast<uint32_t *>(Sh + i * DL_LDS + c) = x;
                    *reinterpret_cast<uint32_t *>(Sl + i * DL_LDS + c) = y;
                    if (i < d && n0 + c < dv) {
                        *reinterpret_cast<uint32_t *>(before + (size_t)i * dv + n0 + c) = x;
                        *reinterpret_cast<uint32_t *>(before + (size_t)(d + i) * dv + n0 + c) = y;
                    }
                }
        dc_wait<1>();
        __syncthreads();
        float acc[3][2][4];                           // three independent chains a column tile: hi hi, hi lo, lo hi
#pragma unroll
        for (int x = 0; x < 3; ++x)
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int c = 0; c < 4; ++c) acc[x][j][c] = 0.f;
#pragma unroll
        for (int kk = 0; kk < D / 16; ++kk) {
            uint32_t a[4], al[4], b0, b1, b2, b3;
            ldmatrix_x4(dc_smem(W1 + a_row * (D + 8) + kk * 16 + a_kk), a[0], a[1], a[2], a[3]);
            ldmatrix_x4(dc_smem(W2 + a_row * (D + 8) + kk * 16 + a_kk), al[0], al[1], al[2], al[3]);
            ldmatrix_x4_trans(dc_smem(Sh + (kk * 16 + v_row) * DL_LDS + v_col), b0, b1, b2, b3);
            mma_bf16(acc[0][0], a, b0, b1);
            mma_bf16(acc[0][1], a, b2, b3);
            mma_bf16(acc[2][0], al, b0, b1);
            mma_bf16(acc[2][1], al, b2, b3);
            ldmatrix_x4_trans(dc_smem(Sl + (kk * 16 + v_row) * DL_LDS + v_col), b0, b1, b2, b3);
            mma_bf16(acc[1][0], a, b0, b1);
            mma_bf16(acc[1][1], a, b2, b3);
        }
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const int i = warp * 16 + g + 8 * hf;
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int c = j * 8 + 2 * tq;
                const float x = u0[hf][j].x - (acc[0][j][2 * hf] + (acc[1][j][2 * hf] + acc[2][j][2 * hf]));
                const float y = u0[hf][j].y - (acc[0][j][2 * hf + 1] + (acc[1][j][2 * hf + 1] + acc[2][j][2 * hf + 1]));
                uint32_t a, b;
                if (i < n && n0 + c < dv) {
                    const size_t o = ((size_t)tb + row0 + i) * p.H * dv + (size_t)h * dv + n0 + c;
                    dc_split2(x, y, a, b);
                    *reinterpret_cast<uint32_t *>(p.u_hi + o) = a;
                    *reinterpret_cast<uint32_t *>(p.u_lo + o) = b;
                }
                dc_split2(x * kf[hf], y * kf[hf], a, b);
                *reinterpret_cast<uint32_t *>(Uh + i * DL_LDS + c) = a;
                *reinterpret_cast<uint32_t *>(Ul + i * DL_LDS + c) = b;
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int mt = warp + 4 * m;
            if (mt * 16 >= D) continue;
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int c = 0; c < 4; ++c) S[m][j][c] *= total;
#pragma unroll
            for (int kk = 0; kk < DC_C / 16; ++kk) {
                uint32_t a[4], b0, b1, b2, b3;
                ldmatrix_x4_trans(dc_smem(Ks + (kk * 16 + t_k) * (D + 8) + mt * 16 + t_m), a[0], a[1], a[2], a[3]);
                ldmatrix_x4_trans(dc_smem(Uh + (kk * 16 + v_row) * DL_LDS + v_col), b0, b1, b2, b3);
                mma_bf16(S[m][0], a, b0, b1);
                mma_bf16(S[m][1], a, b2, b3);
                ldmatrix_x4_trans(dc_smem(Ul + (kk * 16 + v_row) * DL_LDS + v_col), b0, b1, b2, b3);
                mma_bf16(S[m][0], a, b0, b1);
                mma_bf16(S[m][1], a, b2, b3);
            }
        }
        __syncthreads();                              // the stage may be filled again, and the terms in shared memory rewritten
    }
    dc_wait<0>();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int i = (warp + 4 * m) * 16 + g + 8 * (c >> 1), col = n0 + j * 8 + 2 * tq + (c & 1);
                if (i < d && col < dv) st[(size_t)i * dv + col] = S[m][j][c];
            }
}

KESTREL_API int kestrel_delta_steps(const void *act, long long ld_act, const float *partial, int S, long long slice_stride, int ld, int col_beta, int col_a,
                                    const float *A_log, const float *dt_bias, float *q_scale, float *k_scale, float *beta, float *log_decay, int T, int H,
                                    int G, int d, cudaStream_t stream) {
    if (T == 0) return 0;
    KESTREL_REQUIRE(T > 0 && S > 0 && H > 0 && G > 0 && H % G == 0 && d > 0 && d % 2 == 0 && ld_act % 2 == 0 && col_beta >= 0 && col_beta + H <= ld && col_a >= 0 &&
                    col_a + H <= ld, "delta_steps: bad sizes");
    kestrel_launch(delta_steps_kernel, dim3(T), dim3(128), 0, stream, (const __nv_bfloat16 *)act, ld_act, partial, S, (size_t)slice_stride, ld, col_beta, col_a,
                   A_log, dt_bias, q_scale, k_scale, beta, log_decay, H, G, d);
    return kestrel_check_launch("delta_steps");
}

template <int D>
static int dl_launch(const DeltaChunkParams &p, int tiles, int nseq, cudaStream_t stream) {
    const size_t solve = (size_t)DC_C * 68 * 4 + (size_t)DC_C * (D + 8 + 5 * DC_LDN) * 2;
    const size_t scan = (size_t)(2 * 3 * DC_C * (D + 8) + 2 * D * DL_LDS + 2 * DC_C * DL_LDS) * 2;
    static bool attr_set = false;
    if (!attr_set) {
        if (cudaFuncSetAttribute(delta_chunk_solve_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)solve) != cudaSuccess ||
            cudaFuncSetAttribute(delta_chunk_state_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, KESTREL_SMEM_MAX_DYNAMIC) != cudaSuccess)
            return kestrel_fail(-3, "delta_chunks: cannot set the shared memory size");
        attr_set = true;
    }
    kestrel_launch(delta_chunk_solve_kernel<D>, dim3(tiles, p.H), dim3(128), solve, stream, p);
    int rc = kestrel_check_launch("delta_chunk_solve");
    if (rc) return rc;
    const dim3 grid((p.dv + DL_NC - 1) / DL_NC, p.H, nseq);
    kestrel_launch(delta_chunk_state_kernel<D>, grid, dim3(128), kestrel_spread_smem((long)grid.x * grid.y * grid.z, scan), stream, p);
    return kestrel_check_launch("delta_chunk_state");
}

// scratch: tiles H (64 (d + dv) + 68 + d dv) floats
KESTREL_API int kestrel_delta_chunks(const void *act, long long ld_act, int G, const float *q_scale, const float *k_scale, const float *beta,
                                     const float *log_decay, const float *w, float eps, const float *partial, int S, long long slice_stride, int ld, int col_g,
                                     float *state, long long state_stride, long long state_off, const int *cu_seqlens, const int *slots, const int *tile_seq,
                                     const int *tile_row0, const int *first_tile, int tiles, float *scratch, void *u_hi, void *u_lo, void *out, int nseq, int H,
                                     int d, int dv, cudaStream_t stream) {
    if (nseq == 0 || tiles == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && tiles > 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && d > 0 && dv > 0 && d % 8 == 0 && dv % 8 == 0 &&
                    d <= 128 && dv <= 256 && state_off >= 0, "delta_chunks: bad sizes H=%d G=%d d=%d dv=%d", H, G, d, dv);
    KESTREL_REQUIRE(ld_act % 8 == 0 && (((uintptr_t)act | (uintptr_t)scratch | (uintptr_t)u_hi | (uintptr_t)u_lo) & 15) == 0, "delta_chunks: rows on 16-byte boundaries");
    DeltaChunkParams p = {};
    p.act = (const __nv_bfloat16 *)act; p.ld_act = ld_act; p.G = G; p.k_scale = k_scale; p.beta = beta; p.log_decay = log_decay;
    p.cu_seqlens = cu_seqlens; p.slots = slots; p.tile_seq = tile_seq; p.tile_row0 = tile_row0; p.first_tile = first_tile;
    p.state = state; p.state_stride = state_stride; p.state_off = state_off;
    const size_t th = (size_t)tiles * H;
    p.w_hi = (__nv_bfloat16 *)scratch; p.w_lo = p.w_hi + th * DC_C * d;                  // 64 d floats of room together
    p.u0 = scratch + th * DC_C * d;
    p.factors = p.u0 + th * DC_C * dv;
    p.before = (__nv_bfloat16 *)(p.factors + th * 68);
    p.u_hi = (__nv_bfloat16 *)u_hi; p.u_lo = (__nv_bfloat16 *)u_lo; p.H = H; p.d = d; p.dv = dv;
    int rc = d <= 32 ? dl_launch<32>(p, tiles, nseq, stream) : d <= 64 ? dl_launch<64>(p, tiles, nseq, stream) : dl_launch<128>(p, tiles, nseq, stream);
    if (rc) return rc;
    return kestrel_delta_chunks_out(act, ld_act, G, u_hi, u_lo, q_scale, k_scale, log_decay, p.before, w, eps, partial, S, slice_stride, ld, col_g, cu_seqlens,
                                    tile_seq, tile_row0, tiles, out, H, d, dv, stream);
}
