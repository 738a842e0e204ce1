// The recurrence of time_mix.cu - a decay per head, key channel and token, read-out of the old state with a bonus - in chunks of 64
// tokens on the tensor cores.  With E_i the sum of the logarithms of the decays over a chunk's tokens in front of i, per channel, and
// L_j the one that includes j,
//
//   o_i = (r_i e^{E_i}) S + sum_{j < i} (sum_c r_ic k_jc e^{E_ic - L_jc}) v_j + (sum_c r_ic u_c k_ic) v_i
//   S'  = diag(e^{L_n}) S + sum_j (k_j e^{L_n - L_j}) v_j^T
//
// The scores' exponents are sums of logarithms of decays, at most 0, but their two halves are not: e^{-L_j} alone overflows.  So a warp's
// sixteen tokens take the state of the sums in front of THEM as the reference for all earlier sixteens - r_i e^{E_i - ref} and
// k_j e^{ref - L_j} are both at most in size what r and k are, and their product is one on the tensor cores -, its last eight the same way
// for its first eight, and the pairs inside an eight are summed channel by channel with their own exponent in float32.
//
// r, k, v are the bfloat16 operands the projections give; what the decays touch is float32 and enters a product as two bfloat16 terms.
#include "decay_chunks.cuh"
#include <math.h>

struct TimeMixChunkParams {
    const __nv_bfloat16 *r, *k, *v;      // [T, H d]
    const float *log_w;                  // [T, H d]
    const float *u;                      // [H, d]
    const int *cu_seqlens, *slots, *tile_seq, *tile_row0, *first_tile;
    float *state, *scratch, *total;      // scratch [tiles, H, d, d]; total [tiles, H, d] = e^{L_n}
    __nv_bfloat16 *before;               // [tiles, H, 2, d, d]
    long long state_stride, state_off;
    const float *gate;                   // the product whose columns gate_col0 + h d are the gate
    int gate_slices, gate_ld, gate_col0;
    long long gate_stride;
    const float *norm_w;                 // [H d]
    float eps, scale;
    __nv_bfloat16 *out;
    long long ldo;
    int H, d;
};

// r, k, v out of their product in bfloat16, the logarithms of the decays in float32, the request's last h into its slot
__global__ void __launch_bounds__(256)
time_mix_operands_kernel(const float *__restrict__ p, int S, size_t slice_stride, int ld, const float *__restrict__ z, int Sz, size_t z_stride,
                         const float *__restrict__ w0, __nv_bfloat16 *__restrict__ r_out, __nv_bfloat16 *__restrict__ k_out,
                         __nv_bfloat16 *__restrict__ v_out, float *__restrict__ lw_out, int n, const __nv_bfloat16 *__restrict__ h, int width,
                         float *__restrict__ state, size_t state_stride, size_t last_off, const int *__restrict__ seq_of_token,
                         const int *__restrict__ cu_seqlens, const int *__restrict__ slots) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, seq = seq_of_token[t];
    auto sum4 = [&](const float *src, int slices, size_t stride) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int s = 0; s < slices; ++s) {
            const float4 x = *reinterpret_cast<const float4 *>(src + (size_t)s * stride);
            v.x += x.x; v.y += x.y; v.z += x.z; v.w += x.w;
        }
        return v;
    };
    auto put = [](__nv_bfloat16 *dst, const float4 v) { *reinterpret_cast<uint2 *>(dst) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w)); };
    for (int i = 4 * threadIdx.x; i < n; i += 1024) {
        const size_t o = (size_t)t * n + i;
        const float *row = p + (size_t)t * ld + i;
        put(r_out + o, sum4(row, S, slice_stride));
        put(k_out + o, sum4(row + n, S, slice_stride));
        put(v_out + o, sum4(row + 2 * (size_t)n, S, slice_stride));
        float4 y = sum4(z + o, Sz, z_stride);
        const float4 b = *reinterpret_cast<const float4 *>(w0 + i);
        y.x = -expf(y.x + b.x); y.y = -expf(y.y + b.y); y.z = -expf(y.z + b.z); y.w = -expf(y.w + b.w);
        *reinterpret_cast<float4 *>(lw_out + o) = y;
    }
    if (t + 1 == cu_seqlens[seq + 1]) {
        float *last = state + (size_t)slots[seq] * state_stride + last_off;
        for (int i = threadIdx.x; i < width; i += 256) last[i] = __bfloat162float(h[(size_t)t * width + i]);
    }
}

// scratch[tile, h] = sum_j (k_j e^{L_n - L_j}) v_j^T, value columns [64 z, 64 z + 64)
template <int D>
__global__ void __launch_bounds__(128)
time_mix_chunk_kv_kernel(const TimeMixChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t tm_raw[];
    __nv_bfloat16 *Kh = reinterpret_cast<__nv_bfloat16 *>(tm_raw), *Kl = Kh + DC_C * (D + 8), *Vs = Kl + DC_C * (D + 8);
    const int tile = blockIdx.x, h = blockIdx.y, n0 = blockIdx.z * DC_N, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = p.tile_seq[tile], row0 = p.tile_row0[tile], tb = p.cu_seqlens[seq], n = min(DC_C, p.cu_seqlens[seq + 1] - tb - row0);
    const int d = p.d;
    const size_t t0 = (size_t)tb + row0, ld = (size_t)p.H * d;
    for (int idx = tid; idx < DC_C * (DC_N / 8); idx += 128) {
        const int r = idx / (DC_N / 8), c = idx % (DC_N / 8) * 8;
        const bool ok = r < n && n0 + c < d;
        dc_cp16(Vs + r * DC_LDN + c, p.v + (ok ? (t0 + r) * ld + (size_t)h * d + n0 + c : 0), ok);
    }
    dc_commit();
    for (int c = tid; c < D; c += 128) {              // from the chunk's end to its start
        float s = 0.f;
        const size_t base = t0 * ld + (size_t)h * d + c;
        for (int j0 = DC_C - 16; j0 >= 0; j0 -= 16) {
            float lw[16], kk[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                const bool ok = j0 + j < n && c < d;
                lw[j] = ok ? p.log_w[base + (size_t)(j0 + j) * ld] : 0.f;
                kk[j] = ok ? __bfloat162float(p.k[base + (size_t)(j0 + j) * ld]) : 0.f;
            }
#pragma unroll
            for (int j = 15; j >= 0; --j) {
                dc_split(kk[j] * __expf(s), Kh[(j0 + j) * (D + 8) + c], Kl[(j0 + j) * (D + 8) + c]);
                s += lw[j];
            }
        }
        if (c < d && blockIdx.z == 0) p.total[((size_t)tile * p.H + h) * d + c] = expf(s);
    }
    dc_wait<0>();
    __syncthreads();
    const int g = lane >> 2, tq = lane & 3;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    const int a_k = (lane & 7) + (lane >> 4) * 8, a_m = ((lane >> 3) & 1) * 8;
    float *dst = p.scratch + ((size_t)tile * p.H + h) * d * d;
    for (int mt = warp; mt * 16 < d; mt += 4) {
        float acc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[j][c] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DC_C / 16; ++kk) {
            uint32_t a[4], al[4];
            ldmatrix_x4_trans(dc_smem(Kh + (kk * 16 + a_k) * (D + 8) + mt * 16 + a_m), a[0], a[1], a[2], a[3]);
            ldmatrix_x4_trans(dc_smem(Kl + (kk * 16 + a_k) * (D + 8) + mt * 16 + a_m), al[0], al[1], al[2], al[3]);
#pragma unroll
            for (int np = 0; np < DC_N / 16; ++np) {
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
            if (col >= d) continue;
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = mt * 16 + g + 8 * hf;
                if (i < d) *reinterpret_cast<float2 *>(dst + (size_t)i * d + col) = make_float2(acc[j][2 * hf], acc[j][2 * hf + 1]);
            }
        }
    }
}

// Per request and head: the state in front of every chunk, as the two terms its product takes, then the state after the last one.
__global__ void __launch_bounds__(256)
time_mix_chunk_scan_kernel(const TimeMixChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, seq = blockIdx.z, d = p.d, n4 = d * d / 4, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= n4) return;
    const int lo = p.first_tile[seq], hi = p.first_tile[seq + 1], row = 4 * i / d;
    if (lo == hi) return;
    float4 *st = reinterpret_cast<float4 *>(p.state + (size_t)p.slots[seq] * p.state_stride + p.state_off + (size_t)h * d * d) + i;
    const float4 *sc = reinterpret_cast<const float4 *>(p.scratch) + ((size_t)lo * p.H + h) * n4 + i;
    uint2 *bf = reinterpret_cast<uint2 *>(p.before) + ((size_t)lo * p.H + h) * 2 * n4 + i;
    const float *tot = p.total + ((size_t)lo * p.H + h) * d + row;
    const size_t step = (size_t)p.H * n4;
    float4 s = *st;
    for (int c = lo; c < hi; c += 8) {
        float4 kv[8];
        float dec[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (c + u < hi) {
                kv[u] = sc[(size_t)(c - lo + u) * step];
                dec[u] = tot[(size_t)(c - lo + u) * p.H * d];
            }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            if (c + u >= hi) break;
            uint2 a, b;
            dc_split2(s.x, s.y, a.x, b.x);
            dc_split2(s.z, s.w, a.y, b.y);
            bf[(size_t)(c - lo + u) * 2 * step] = a;
            bf[(size_t)(c - lo + u) * 2 * step + n4] = b;
            s.x = fmaf(dec[u], s.x, kv[u].x);
            s.y = fmaf(dec[u], s.y, kv[u].y);
            s.z = fmaf(dec[u], s.z, kv[u].z);
            s.w = fmaf(dec[u], s.w, kv[u].w);
        }
    }
    *st = s;
}

// A chunk's outputs of a head: warp w has tokens 16 w .. 16 w + 15; NS slices of 64 value columns.
template <int D, int NS>
__global__ void __launch_bounds__(128)
time_mix_chunk_out_kernel(const TimeMixChunkParams p) {
    constexpr int LDL = D + 4;
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t tm_raw[];
    float *Ls = reinterpret_cast<float *>(tm_raw);                             // [65][LDL]: row i = E_i, row i + 1 = L_i
    float *us = Ls + (DC_C + 1) * LDL;                                         // [D]
    __nv_bfloat16 *Rs = reinterpret_cast<__nv_bfloat16 *>(us + D), *Ks = Rs + DC_C * (D + 8), *Vs = Ks + DC_C * (D + 8);
    __nv_bfloat16 *Sh = Vs + DC_C * DC_LDN, *Sl = Sh + D * DC_LDN;
    const int tile = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = p.tile_seq[tile], row0 = p.tile_row0[tile], tb = p.cu_seqlens[seq], n = min(DC_C, p.cu_seqlens[seq + 1] - tb - row0);
    const int d = p.d, k_steps = (d + 15) / 16;
    const size_t t0 = (size_t)tb + row0, ld = (size_t)p.H * d;
    const __nv_bfloat16 *st = p.before + ((size_t)tile * p.H + h) * 2 * d * d;
    auto load_slice = [&](int n0) {
        for (int idx = tid; idx < DC_C * (DC_N / 8); idx += 128) {
            const int r = idx / (DC_N / 8), c = idx % (DC_N / 8) * 8;
            const bool ok = r < n && n0 + c < d;
            dc_cp16(Vs + r * DC_LDN + c, p.v + (ok ? (t0 + r) * ld + (size_t)h * d + n0 + c : 0), ok);
        }
        for (int idx = tid; idx < D * (DC_N / 8); idx += 128) {
            const int i = idx / (DC_N / 8), c = idx % (DC_N / 8) * 8;
            const bool ok = i < d && n0 + c < d;
            const size_t off = ok ? (size_t)i * d + n0 + c : 0;
            dc_cp16(Sh + i * DC_LDN + c, st + off, ok);
            dc_cp16(Sl + i * DC_LDN + c, st + (size_t)d * d + off, ok);
        }
        dc_commit();
    };
    dc_load_rows<D>(Rs, p.r + t0 * ld + (size_t)h * d, ld, n, d, tid);
    dc_load_rows<D>(Ks, p.k + t0 * ld + (size_t)h * d, ld, n, d, tid);
    dc_commit();
    load_slice(0);                                    // under the scores
    // the running sums, in base-2 units: half a chunk's tokens of a channel a thread, all of its loads in flight; the second half
    // then gets the first one's total
    for (int idx = tid; idx < 2 * D; idx += 128) {
        const int c = idx % D, j0 = idx / D * (DC_C / 2);
        const float *src = p.log_w + (t0 + j0) * ld + (size_t)h * d + c;
        float lw[DC_C / 2], s = 0.f;
#pragma unroll
        for (int j = 0; j < DC_C / 2; ++j) lw[j] = j0 + j < n && c < d ? src[(size_t)j * ld] : 0.f;
#pragma unroll
        for (int j = 0; j < DC_C / 2; ++j) {
            s += lw[j];
            Ls[(j0 + j + 1) * LDL + c] = s * 1.4426950408889634f;
        }
        if (j0 == 0) {
            us[c] = c < d ? p.u[(size_t)h * d + c] : 0.f;
            Ls[c] = 0.f;
        }
    }
    __syncthreads();
    for (int idx = tid; idx < DC_C / 2 * D; idx += 128) Ls[(DC_C / 2 + 1 + idx / D) * LDL + idx % D] += Ls[DC_C / 2 * LDL + idx % D];
    dc_wait<1>();
    __syncthreads();
    const int g = lane >> 2, tq = lane & 3;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    const int i0 = warp * 16 + g, i1 = i0 + 8;        // this lane's two rows
    auto pair = [](const __nv_bfloat16 *q) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(q)); };
    // two neighbouring channels of a row of r, times 2^{E_i - ref}, in two terms (ref null: nothing is subtracted)
    auto r_terms = [&](int i, int c, const float *ref, uint32_t &hi, uint32_t &lo) {
        const float2 r = pair(Rs + i * (D + 8) + c), e = *reinterpret_cast<const float2 *>(Ls + i * LDL + c);
        const float2 m = ref ? *reinterpret_cast<const float2 *>(ref + c) : make_float2(0.f, 0.f);
        dc_split2(r.x * fast_exp2(e.x - m.x), r.y * fast_exp2(e.y - m.y), hi, lo);
    };
    uint32_t ph[DC_C / 16][4], pl[DC_C / 16][4];      // the scores as two terms, in the layout of an A operand
    {
        float s[DC_C / 8][4];
#pragma unroll
        for (int j = 0; j < DC_C / 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[j][c] = 0.f;
        // two neighbouring channels of a key, times 2^{ref - L_j}, in two terms
        auto k_terms = [&](int j, int c, const float *ref, uint32_t &hi, uint32_t &lo) {
            const float2 k = pair(Ks + j * (D + 8) + c), l = *reinterpret_cast<const float2 *>(Ls + (j + 1) * LDL + c),
                         m = *reinterpret_cast<const float2 *>(ref + c);
            dc_split2(k.x * fast_exp2(m.x - l.x), k.y * fast_exp2(m.y - l.y), hi, lo);
        };
        const float *ref = Ls + warp * 16 * LDL, *mid = ref + 8 * LDL;
        if (warp > 0) {                               // keys of the earlier sixteens (the branch is a warp's)
            for (int kk = 0; kk < k_steps; ++kk) {
                uint32_t a[4], al[4];
                r_terms(i0, kk * 16 + 2 * tq, ref, a[0], al[0]);
                r_terms(i1, kk * 16 + 2 * tq, ref, a[1], al[1]);
                r_terms(i0, kk * 16 + 2 * tq + 8, ref, a[2], al[2]);
                r_terms(i1, kk * 16 + 2 * tq + 8, ref, a[3], al[3]);
#pragma unroll
                for (int jt = 0; jt < 6; ++jt) {
                    if (jt >= 2 * warp) continue;
                    uint32_t b[2], bl[2];
#pragma unroll
                    for (int x = 0; x < 2; ++x) k_terms(jt * 8 + g, kk * 16 + 2 * tq + 8 * x, ref, b[x], bl[x]);
                    mma_bf16(s[jt], a, b[0], b[1]);
                    mma_bf16(s[jt], a, bl[0], bl[1]);
                    mma_bf16(s[jt], al, b[0], b[1]);
                }
            }
        }
        // inside the sixteen: the last eight tokens with the first eight once more as a product, the sums in front of the eighth as the
        // reference (the rows of the first eight stay out of it)
        float x8[4] = {0.f, 0.f, 0.f, 0.f};
        for (int kk = 0; kk < k_steps; ++kk) {
            uint32_t a[4] = {0, 0, 0, 0}, al[4] = {0, 0, 0, 0}, b[2], bl[2];
            r_terms(i1, kk * 16 + 2 * tq, mid, a[1], al[1]);
            r_terms(i1, kk * 16 + 2 * tq + 8, mid, a[3], al[3]);
#pragma unroll
            for (int x = 0; x < 2; ++x) k_terms(warp * 16 + g, kk * 16 + 2 * tq + 8 * x, mid, b[x], bl[x]);
            mma_bf16(x8, a, b[0], b[1]);
            mma_bf16(x8, a, bl[0], bl[1]);
            mma_bf16(x8, al, b[0], b[1]);
        }
        // and the pairs inside each eight: this lane's row i0 + 8 a with columns j = 16 warp + 8 a + 2 tq + {0, 1}
        float q[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
        const int jb = warp * 16 + 2 * tq;
        for (int c = 0; c < d; c += 2) {
            const float2 uu = *reinterpret_cast<const float2 *>(us + c);
#pragma unroll
            for (int a = 0; a < 2; ++a) {
                const int i = i0 + 8 * a;
                const float2 r = pair(Rs + i * (D + 8) + c), e = *reinterpret_cast<const float2 *>(Ls + i * LDL + c);
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    const int j = jb + 8 * a + b;
                    const float2 k = pair(Ks + j * (D + 8) + c), l = *reinterpret_cast<const float2 *>(Ls + (j + 1) * LDL + c);
                    const float fx = i == j ? uu.x : fast_exp2(fminf(e.x - l.x, 0.f)), fy = i == j ? uu.y : fast_exp2(fminf(e.y - l.y, 0.f));
                    q[a][b] = fmaf(r.x * k.x, fx, fmaf(r.y * k.y, fy, q[a][b]));
                }
            }
        }
#pragma unroll
        for (int jt = 0; jt < DC_C / 8; ++jt) {
            if ((jt >> 1) != warp) continue;
            const int a = jt & 1;                     // the eight this column tile belongs to
#pragma unroll
            for (int b = 0; b < 2; ++b) {
                if (a == 0) {
                    s[jt][b] = i0 >= jb + b ? q[0][b] : 0.f;
                    s[jt][2 + b] = x8[2 + b];
                } else {
                    s[jt][b] = 0.f;
                    s[jt][2 + b] = i1 >= jb + 8 + b ? q[1][b] : 0.f;
                }
            }
        }
#pragma unroll
        for (int jp = 0; jp < DC_C / 16; ++jp)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int jt = 2 * jp + (e >> 1);
                dc_split2(s[jt][2 * (e & 1)], s[jt][2 * (e & 1) + 1], ph[jp][e], pl[jp][e]);
            }
    }
    float o[NS][DC_N / 8][4];
#pragma unroll
    for (int ns = 0; ns < NS; ++ns) {
        if (ns > 0) {
            __syncthreads();                          // everyone has left the slice before
            load_slice(ns * DC_N);
        }
        dc_wait<0>();
        __syncthreads();
        float (&oo)[DC_N / 8][4] = o[ns];
#pragma unroll
        for (int j = 0; j < DC_N / 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) oo[j][c] = 0.f;
        for (int kk = 0; kk < k_steps; ++kk) {
            uint32_t a[4], al[4];
            r_terms(i0, kk * 16 + 2 * tq, nullptr, a[0], al[0]);
            r_terms(i1, kk * 16 + 2 * tq, nullptr, a[1], al[1]);
            r_terms(i0, kk * 16 + 2 * tq + 8, nullptr, a[2], al[2]);
            r_terms(i1, kk * 16 + 2 * tq + 8, nullptr, a[3], al[3]);
#pragma unroll
            for (int np = 0; np < DC_N / 16; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(dc_smem(Sh + (kk * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], a, b0, b1);
                mma_bf16(oo[2 * np + 1], a, b2, b3);
                mma_bf16(oo[2 * np], al, b0, b1);
                mma_bf16(oo[2 * np + 1], al, b2, b3);
                ldmatrix_x4_trans(dc_smem(Sl + (kk * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], a, b0, b1);
                mma_bf16(oo[2 * np + 1], a, b2, b3);
            }
        }
#pragma unroll
        for (int jp = 0; jp < DC_C / 16; ++jp) {
            if (jp > warp) continue;
#pragma unroll
            for (int np = 0; np < DC_N / 16; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(dc_smem(Vs + (jp * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], ph[jp], b0, b1);
                mma_bf16(oo[2 * np + 1], ph[jp], b2, b3);
                mma_bf16(oo[2 * np], pl[jp], b0, b1);
                mma_bf16(oo[2 * np + 1], pl[jp], b2, b3);
            }
        }
    }
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        const int i = i0 + 8 * hf;
        float ss = 0.f;
#pragma unroll
        for (int ns = 0; ns < NS; ++ns)
#pragma unroll
            for (int j = 0; j < DC_N / 8; ++j) ss = fmaf(o[ns][j][2 * hf], o[ns][j][2 * hf], fmaf(o[ns][j][2 * hf + 1], o[ns][j][2 * hf + 1], ss));
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        if (i >= n) continue;
        const float rn = (1.0f / sqrtf(ss / (float)d + p.eps)) * p.scale;
        const size_t gate_row = (t0 + i) * p.gate_ld + p.gate_col0 + (size_t)h * d;
        __nv_bfloat16 *dst = p.out + (t0 + i) * p.ldo + (size_t)h * d;
        const float *w = p.norm_w + (size_t)h * d;
        float2 z[NS][DC_N / 8];
#pragma unroll
        for (int ns = 0; ns < NS; ++ns)
#pragma unroll
            for (int j = 0; j < DC_N / 8; ++j) z[ns][j] = make_float2(0.f, 0.f);
        for (int s = 0; s < p.gate_slices; ++s)
#pragma unroll
            for (int ns = 0; ns < NS; ++ns)
#pragma unroll
                for (int j = 0; j < DC_N / 8; ++j) {
                    const int col = ns * DC_N + j * 8 + 2 * tq;
                    if (col >= d) continue;
                    const float2 x = *reinterpret_cast<const float2 *>(p.gate + (size_t)s * p.gate_stride + gate_row + col);
                    z[ns][j].x += x.x;
                    z[ns][j].y += x.y;
                }
#pragma unroll
        for (int ns = 0; ns < NS; ++ns)
#pragma unroll
            for (int j = 0; j < DC_N / 8; ++j) {
                const int col = ns * DC_N + j * 8 + 2 * tq;
                if (col >= d) continue;
                const float z0 = z[ns][j].x, z1 = z[ns][j].y;
                *reinterpret_cast<uint32_t *>(dst + col) = pack_bf16(o[ns][j][2 * hf] * rn * w[col] * (z0 / (1.0f + __expf(-z0))),
                                                                     o[ns][j][2 * hf + 1] * rn * w[col + 1] * (z1 / (1.0f + __expf(-z1))));
            }
    }
}

template <int D, int NS>
static int tm_launch(const TimeMixChunkParams &p, int tiles, int nseq, cudaStream_t stream) {
    const size_t kv_smem = (size_t)DC_C * (2 * (D + 8) + DC_LDN) * 2;
    const size_t out_smem = (size_t)((DC_C + 1) * (D + 4) + D) * 4 + (size_t)(DC_C * (2 * (D + 8) + DC_LDN) + 2 * D * DC_LDN) * 2;
    static bool attr_set = false;
    if (!attr_set) {
        if (cudaFuncSetAttribute(time_mix_chunk_kv_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kv_smem) != cudaSuccess ||
            cudaFuncSetAttribute(time_mix_chunk_out_kernel<D, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem) != cudaSuccess)
            return kestrel_fail(-3, "time_mix_chunks: cannot set the shared memory size");
        attr_set = true;
    }
    kestrel_launch(time_mix_chunk_kv_kernel<D>, dim3(tiles, p.H, NS), dim3(128), kv_smem, stream, p);
    int rc = kestrel_check_launch("time_mix_chunk_kv");
    if (rc) return rc;
    kestrel_launch(time_mix_chunk_scan_kernel, dim3((p.d * p.d / 4 + 255) / 256, p.H, nseq), dim3(256), 0, stream, p);
    if ((rc = kestrel_check_launch("time_mix_chunk_scan"))) return rc;
    kestrel_launch(time_mix_chunk_out_kernel<D, NS>, dim3(tiles, p.H), dim3(128), out_smem, stream, p);
    return kestrel_check_launch("time_mix_chunk_out");
}

// operands: 3 T H d bfloat16; log_w: T H d floats; scratch: tiles H (2 d d + d) floats
KESTREL_API int kestrel_time_mix_chunks(const float *partial, int S, long long slice_stride, int ld, const float *z, int Sz, long long z_stride, const float *w0,
                                        const float *u, const float *norm_w, float eps, float scale, const void *h, int width, float *state,
                                        long long state_stride, long long state_off, long long last_off, const int *seq_of_token, const int *cu_seqlens,
                                        const int *slots, const int *tile_seq, const int *tile_row0, const int *first_tile, int tiles, void *operands,
                                        float *log_w, float *scratch, void *out, long long ldo, int T, int nseq, int H, int d, cudaStream_t stream) {
    if (T == 0 || nseq == 0 || tiles == 0) return 0;
    const int n = H * d;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && tiles > 0 && H > 0 && H <= 65535 && d > 0 && d % 8 == 0 && d <= 128 && S > 0 && Sz > 0, "time_mix_chunks: bad sizes H=%d d=%d", H, d);
    KESTREL_REQUIRE(ld >= 4 * n && ld % 4 == 0 && slice_stride % 4 == 0 && z_stride % 4 == 0 && state_stride % 4 == 0 && state_off % 4 == 0 && ldo % 2 == 0 &&
                    (((uintptr_t)partial | (uintptr_t)z | (uintptr_t)w0 | (uintptr_t)state | (uintptr_t)operands | (uintptr_t)log_w | (uintptr_t)scratch) & 15) == 0 &&
                    ((uintptr_t)out & 3) == 0, "time_mix_chunks: the products, the state's place or the output do not fit");
    __nv_bfloat16 *r = (__nv_bfloat16 *)operands, *k = r + (size_t)T * n, *v = k + (size_t)T * n;
    kestrel_launch(time_mix_operands_kernel, dim3(T), dim3(256), 0, stream, partial, S, (size_t)slice_stride, ld, z, Sz, (size_t)z_stride, w0, r, k, v, log_w, n,
                   (const __nv_bfloat16 *)h, width, state, (size_t)state_stride, (size_t)last_off, seq_of_token, cu_seqlens, slots);
    int rc = kestrel_check_launch("time_mix_operands");
    if (rc) return rc;
    TimeMixChunkParams p = {};
    p.r = r; p.k = k; p.v = v; p.log_w = log_w; p.u = u; p.cu_seqlens = cu_seqlens; p.slots = slots; p.tile_seq = tile_seq; p.tile_row0 = tile_row0;
    p.first_tile = first_tile; p.state = state; p.state_stride = state_stride; p.state_off = state_off;
    const size_t m = (size_t)tiles * H * d * d;
    p.scratch = scratch; p.before = (__nv_bfloat16 *)(scratch + m); p.total = scratch + 2 * m;
    p.gate = partial; p.gate_slices = S; p.gate_ld = ld; p.gate_col0 = 3 * n; p.gate_stride = slice_stride;
    p.norm_w = norm_w; p.eps = eps; p.scale = scale; p.out = (__nv_bfloat16 *)out; p.ldo = ldo; p.H = H; p.d = d;
    if (d <= 32) return tm_launch<32, 1>(p, tiles, nseq, stream);
    if (d <= 64) return tm_launch<64, 1>(p, tiles, nseq, stream);
    return tm_launch<128, 2>(p, tiles, nseq, stream);
}
