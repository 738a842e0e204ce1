// Recurrences with a scalar decay per head and token, in chunks of 64 tokens on the tensor cores:
//
//   S_t = exp(a_t) S_{t-1} + s_t k_t v_t^T,      o_t = S_t^T q_t            a <= 0; s a step size
//
// With L_i the sum of a over a chunk's tokens up to i,
//
//   o_i = exp(L_i) S^T q_i + sum_{j <= i} exp(L_i - L_j) s_j (q_i . k_j) v_j,      S' = exp(L_n) S + sum_j exp(L_n - L_j) s_j k_j v_j^T
//
// chunk_kv makes every chunk's sum over k_j v_j^T, chunk_scan runs a request's chunks in order and leaves the state in front of each,
// chunk_out makes the outputs and what follows them up to the output product.  q, k, v are bfloat16 operands; a query or key may carry
// a float32 factor per token (what makes it a unit vector), which multiplies the scores.  All that the recurrence makes itself - decays,
// steps, weighted values, masked scores, states - is float32 and enters a product as two bfloat16 terms (16 bits of mantissa).
//
// chunk_out has two ends:  0  y = (o + D v) silu(z), float32                          (state-space mixer; its norm spans heads)
//                          1  y = norm per head(o) * w * silu(g), in the storage type   (delta rule, whose v are what its writes left)
#include "decay_chunks.cuh"
#include <math.h>

struct DecayChunkParams {
    const __nv_bfloat16 *q, *k, *v, *v_lo;       // rows of a token; v_lo: the values' second terms, or null
    long long ldq, ldk, ldv;
    int group;                                   // value heads per query/key head
    const float *q_scale, *k_scale;              // [T, H / group], or null
    const float *log_decay, *step;               // [T, H]; step null: 1
    const int *cu_seqlens, *slots, *tile_seq, *tile_row0, *first_tile;
    float *state, *scratch, *total;              // scratch [tiles, H, d, dv]: the chunks' sums; total [tiles, H]: exp(L_n)
    __nv_bfloat16 *before;                       // [tiles, H, 2, d, dv]: the states in front of the chunks, as two terms
    long long state_stride, state_off;
    const float *gate;                           // the fused product with z, or g
    int gate_slices, gate_ld, gate_col0;
    long long gate_stride;
    const float *D;                              // end 0: [H]
    float *y;                                    //        [T, H dv]
    const float *w;                              // end 1: [dv]
    float eps;
    __nv_bfloat16 *out;                          //        [T, H dv]
    int H, d, dv;
};

// scratch[tile, h] = sum_j exp(L_n - L_j) s_j k_j v_j^T, columns [64 z, 64 z + 64)
template <int D>
__global__ void __launch_bounds__(128)
decay_chunk_kv_kernel(const DecayChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t dc_raw[];
    __nv_bfloat16 *Ks = reinterpret_cast<__nv_bfloat16 *>(dc_raw), *Vh = Ks + DC_C * (D + 8), *Vl = Vh + DC_C * DC_LDN;
    __shared__ float L[DC_C], wt[DC_C];
    const int tile = blockIdx.x, h = blockIdx.y, n0 = blockIdx.z * DC_N, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = p.tile_seq[tile], row0 = p.tile_row0[tile], tb = p.cu_seqlens[seq], n = min(DC_C, p.cu_seqlens[seq + 1] - tb - row0);
    const int d = p.d, dv = p.dv;
    const size_t t0 = (size_t)tb + row0;
    dc_load_rows<D>(Ks, p.k + t0 * p.ldk + (size_t)(h / p.group) * d, p.ldk, n, d, tid);
    dc_commit();
    dc_running_sums(L, p.log_decay + t0 * p.H + h, p.H, n, tid);
    __syncthreads();
    if (tid < DC_C) {
        float x = tid < n ? __expf(L[DC_C - 1] - L[tid]) : 0.f;
        if (tid < n && p.step) x *= p.step[(t0 + tid) * p.H + h];
        if (tid < n && p.k_scale) x *= p.k_scale[(t0 + tid) * (p.H / p.group) + h / p.group];
        wt[tid] = x;
    }
    if (tid == 0 && blockIdx.z == 0) p.total[(size_t)tile * p.H + h] = expf(L[DC_C - 1]);
    __syncthreads();
    for (int idx = tid; idx < DC_C * (DC_N / 2); idx += 128) {
        const int r = idx / (DC_N / 2), c = idx % (DC_N / 2) * 2;
        uint32_t hi = 0, lo = 0;
        if (r < n && n0 + c < dv) {
            const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162 *>(p.v + (t0 + r) * p.ldv + (size_t)h * dv + n0 + c);
            dc_split2(__bfloat162float(x.x) * wt[r], __bfloat162float(x.y) * wt[r], hi, lo);
        }
        *reinterpret_cast<uint32_t *>(Vh + r * DC_LDN + c) = hi;
        *reinterpret_cast<uint32_t *>(Vl + r * DC_LDN + c) = lo;
    }
    dc_wait<0>();
    __syncthreads();
    const int g = lane >> 2, tq = lane & 3;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    const int a_k = (lane & 7) + (lane >> 4) * 8, a_m = ((lane >> 3) & 1) * 8;           // K^T fragments: rows of memory are tokens
    float *dst = p.scratch + ((size_t)tile * p.H + h) * d * dv;
    for (int mt = warp; mt * 16 < d; mt += 4) {
        float acc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[j][c] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DC_C / 16; ++kk) {
            uint32_t a[4];
            ldmatrix_x4_trans(dc_smem(Ks + (kk * 16 + a_k) * (D + 8) + mt * 16 + a_m), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int np = 0; np < DC_N / 16; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(dc_smem(Vh + (kk * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(acc[2 * np], a, b0, b1);
                mma_bf16(acc[2 * np + 1], a, b2, b3);
                ldmatrix_x4_trans(dc_smem(Vl + (kk * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(acc[2 * np], a, b0, b1);
                mma_bf16(acc[2 * np + 1], a, b2, b3);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int col = n0 + j * 8 + 2 * tq;
            if (col >= dv) continue;
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int i = mt * 16 + g + 8 * hf;
                if (i < d) *reinterpret_cast<float2 *>(dst + (size_t)i * dv + col) = make_float2(acc[j][2 * hf], acc[j][2 * hf + 1]);
            }
        }
    }
}

// Per request and head: the state in front of every chunk, as the two terms its product takes, then the state after the last one.
__global__ void __launch_bounds__(256)
decay_chunk_scan_kernel(const DecayChunkParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, seq = blockIdx.z, n4 = p.d * p.dv / 4, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= n4) return;
    const int lo = p.first_tile[seq], hi = p.first_tile[seq + 1];
    if (lo == hi) return;
    float4 *st = reinterpret_cast<float4 *>(p.state + (size_t)p.slots[seq] * p.state_stride + p.state_off + (size_t)h * p.d * p.dv) + i;
    const float4 *sc = reinterpret_cast<const float4 *>(p.scratch) + ((size_t)lo * p.H + h) * n4 + i;
    uint2 *bf = reinterpret_cast<uint2 *>(p.before) + ((size_t)lo * p.H + h) * 2 * n4 + i;
    const float *tot = p.total + (size_t)lo * p.H + h;
    const size_t step = (size_t)p.H * n4;
    float4 s = *st;
    for (int c = lo; c < hi; c += 8) {
        float4 kv[8];
        float dec[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (c + u < hi) {
                kv[u] = sc[(size_t)(c - lo + u) * step];
                dec[u] = tot[(size_t)(c - lo + u) * p.H];
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
template <int D, int NS, int END>
__global__ void __launch_bounds__(128)
decay_chunk_out_kernel(const DecayChunkParams p) {
    constexpr bool TWO = END == 1;                    // values in two terms
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) uint8_t dc_raw[];
    __nv_bfloat16 *Qs = reinterpret_cast<__nv_bfloat16 *>(dc_raw), *Ks = Qs + DC_C * (D + 8), *Vs = Ks + DC_C * (D + 8);
    __nv_bfloat16 *Vt = Vs + DC_C * DC_LDN, *Sh = Vt + (TWO ? DC_C * DC_LDN : 0), *Sl = Sh + D * DC_LDN;
    __shared__ float L[DC_C], wt[DC_C], qs[DC_C];
    const int tile = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seq = p.tile_seq[tile], row0 = p.tile_row0[tile], tb = p.cu_seqlens[seq], n = min(DC_C, p.cu_seqlens[seq + 1] - tb - row0);
    const int d = p.d, dv = p.dv, k_steps = (d + 15) / 16, hk = h / p.group, G = p.H / p.group;
    const size_t t0 = (size_t)tb + row0;
    const __nv_bfloat16 *st = p.before + ((size_t)tile * p.H + h) * 2 * d * dv;
    auto load_slice = [&](int n0) {
        for (int idx = tid; idx < DC_C * (DC_N / 8); idx += 128) {
            const int r = idx / (DC_N / 8), c = idx % (DC_N / 8) * 8;
            const bool ok = r < n && n0 + c < dv;
            const size_t off = ok ? (t0 + r) * p.ldv + (size_t)h * dv + n0 + c : 0;
            dc_cp16(Vs + r * DC_LDN + c, p.v + off, ok);
            if (TWO) dc_cp16(Vt + r * DC_LDN + c, p.v_lo + off, ok);
        }
        for (int idx = tid; idx < D * (DC_N / 8); idx += 128) {
            const int i = idx / (DC_N / 8), c = idx % (DC_N / 8) * 8;
            const bool ok = i < d && n0 + c < dv;
            const size_t off = ok ? (size_t)i * dv + n0 + c : 0;
            dc_cp16(Sh + i * DC_LDN + c, st + off, ok);
            dc_cp16(Sl + i * DC_LDN + c, st + (size_t)d * dv + off, ok);
        }
        dc_commit();
    };
    dc_load_rows<D>(Qs, p.q + t0 * p.ldq + (size_t)hk * d, p.ldq, n, d, tid);
    dc_load_rows<D>(Ks, p.k + t0 * p.ldk + (size_t)hk * d, p.ldk, n, d, tid);
    dc_commit();
    load_slice(0);                                    // under the scores
    dc_running_sums(L, p.log_decay + t0 * p.H + h, p.H, n, tid);
    if (tid >= 64) {
        const int j = tid - 64;
        float x = j < n ? 1.f : 0.f;
        if (j < n && p.step) x *= p.step[(t0 + j) * p.H + h];
        if (j < n && p.k_scale) x *= p.k_scale[(t0 + j) * G + hk];
        wt[j] = x;
        qs[j] = j < n && p.q_scale ? p.q_scale[(t0 + j) * G + hk] : 1.f;
    }
    dc_wait<1>();
    __syncthreads();
    const int g = lane >> 2, tq = lane & 3;
    const int a_row = warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, a_k = (lane >> 4) * 8;
    const int b_row = (lane & 7) + (lane >> 4) * 8, b_k = ((lane >> 3) & 1) * 8;
    const int v_row = (lane & 7) + ((lane >> 3) & 1) * 8, v_col = (lane >> 4) * 8;
    // the scores of this warp's tokens with the chunk's, decayed and masked, as two terms in the layout of an A operand
    uint32_t ph[DC_C / 16][4], pl[DC_C / 16][4];
    {
        float s[DC_C / 8][4];
#pragma unroll
        for (int j = 0; j < DC_C / 8; ++j)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[j][c] = 0.f;
        for (int kk = 0; kk < k_steps; ++kk) {
            uint32_t a[4];
            ldmatrix_x4(dc_smem(Qs + a_row * (D + 8) + kk * 16 + a_k), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int jp = 0; jp < DC_C / 16; ++jp) {
                if (jp > warp) continue;              // keys behind the warp's last token
                uint32_t b00, b01, b10, b11;
                ldmatrix_x4(dc_smem(Ks + (jp * 16 + b_row) * (D + 8) + kk * 16 + b_k), b00, b01, b10, b11);
                mma_bf16(s[2 * jp], a, b00, b01);
                mma_bf16(s[2 * jp + 1], a, b10, b11);
            }
        }
#pragma unroll
        for (int jp = 0; jp < DC_C / 16; ++jp)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                // register e of the operand: row g (+ 8), keys 2 tq (+ 8)
                const int jt = 2 * jp + (e >> 1), i = warp * 16 + g + 8 * (e & 1), j = jt * 8 + 2 * tq;
                const float x0 = i >= j ? s[jt][2 * (e & 1)] * (__expf(L[i] - L[j]) * wt[j]) : 0.f;
                const float x1 = i > j ? s[jt][2 * (e & 1) + 1] * (__expf(L[i] - L[j + 1]) * wt[j + 1]) : 0.f;
                dc_split2(x0, x1, ph[jp][e], pl[jp][e]);
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
            uint32_t a[4];
            ldmatrix_x4(dc_smem(Qs + a_row * (D + 8) + kk * 16 + a_k), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int np = 0; np < DC_N / 16; ++np) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(dc_smem(Sh + (kk * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], a, b0, b1);
                mma_bf16(oo[2 * np + 1], a, b2, b3);
                ldmatrix_x4_trans(dc_smem(Sl + (kk * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                mma_bf16(oo[2 * np], a, b0, b1);
                mma_bf16(oo[2 * np + 1], a, b2, b3);
            }
        }
        const float g0 = __expf(L[warp * 16 + g]), g1 = __expf(L[warp * 16 + g + 8]);
#pragma unroll
        for (int j = 0; j < DC_N / 8; ++j) {
            oo[j][0] *= g0;
            oo[j][1] *= g0;
            oo[j][2] *= g1;
            oo[j][3] *= g1;
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
                if (TWO) {
                    ldmatrix_x4_trans(dc_smem(Vt + (jp * 16 + v_row) * DC_LDN + np * 16 + v_col), b0, b1, b2, b3);
                    mma_bf16(oo[2 * np], ph[jp], b0, b1);
                    mma_bf16(oo[2 * np + 1], ph[jp], b2, b3);
                }
            }
        }
        if (END == 0) {                               // + D v while the slice's values are in shared memory
            const float Dh = p.D[h];
#pragma unroll
            for (int j = 0; j < DC_N / 8; ++j)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162 *>(Vs + (warp * 16 + g + 8 * hf) * DC_LDN + j * 8 + 2 * tq);
                    oo[j][2 * hf] = fmaf(Dh, __bfloat162float(x.x), oo[j][2 * hf]);
                    oo[j][2 * hf + 1] = fmaf(Dh, __bfloat162float(x.y), oo[j][2 * hf + 1]);
                }
        }
    }
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
        const int i = warp * 16 + g + 8 * hf;
        float rn = 1.f;
        if (END == 1) {                               // the head's norm (columns beyond dv are zero)
            const float sc = qs[i];
            float ss = 0.f;
#pragma unroll
            for (int ns = 0; ns < NS; ++ns)
#pragma unroll
                for (int j = 0; j < DC_N / 8; ++j) {
                    o[ns][j][2 * hf] *= sc;
                    o[ns][j][2 * hf + 1] *= sc;
                    ss = fmaf(o[ns][j][2 * hf], o[ns][j][2 * hf], fmaf(o[ns][j][2 * hf + 1], o[ns][j][2 * hf + 1], ss));
                }
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            rn = 1.0f / sqrtf(ss / (float)dv + p.eps);
        }
        if (i >= n) continue;
        const size_t gate_row = (t0 + i) * p.gate_ld + p.gate_col0 + (size_t)h * dv, row = (t0 + i) * p.H * dv + (size_t)h * dv;
        float2 z[NS][DC_N / 8];                       // all of a row's gate logits in flight at once
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
                    if (col >= dv) continue;
                    const float2 x = *reinterpret_cast<const float2 *>(p.gate + (size_t)s * p.gate_stride + gate_row + col);
                    z[ns][j].x += x.x;
                    z[ns][j].y += x.y;
                }
#pragma unroll
        for (int ns = 0; ns < NS; ++ns)
#pragma unroll
            for (int j = 0; j < DC_N / 8; ++j) {
                const int col = ns * DC_N + j * 8 + 2 * tq;
                if (col >= dv) continue;
                const float z0 = z[ns][j].x, z1 = z[ns][j].y, a0 = z0 / (1.0f + __expf(-z0)), a1 = z1 / (1.0f + __expf(-z1));
                if (END == 0) {
                    *reinterpret_cast<float2 *>(p.y + row + col) = make_float2(o[ns][j][2 * hf] * a0, o[ns][j][2 * hf + 1] * a1);
                } else {
                    *reinterpret_cast<uint32_t *>(p.out + row + col) =
                        pack_bf16(o[ns][j][2 * hf] * rn * p.w[col] * a0, o[ns][j][2 * hf + 1] * rn * p.w[col + 1] * a1);
                }
            }
    }
}

KESTREL_API int kestrel_decay_chunk_tokens(void) { return DC_C; }

template <int D>
static int dc_kv_scan(const DecayChunkParams &p, int tiles, int nseq, cudaStream_t stream) {
    const size_t smem = (size_t)DC_C * (D + 8 + 2 * DC_LDN) * 2;
    static bool attr_set = false;
    if (!attr_set && cudaFuncSetAttribute(decay_chunk_kv_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return kestrel_fail(-3, "decay_chunks: cannot set the shared memory size");
    attr_set = true;
    kestrel_launch(decay_chunk_kv_kernel<D>, dim3(tiles, p.H, (p.dv + DC_N - 1) / DC_N), dim3(128), smem, stream, p);
    int rc = kestrel_check_launch("decay_chunk_kv");
    if (rc) return rc;
    kestrel_launch(decay_chunk_scan_kernel, dim3((p.d * p.dv / 4 + 255) / 256, p.H, nseq), dim3(256), 0, stream, p);
    return kestrel_check_launch("decay_chunk_scan");
}

template <int D, int NS, int END>
static int dc_out(const DecayChunkParams &p, int tiles, cudaStream_t stream) {
    const size_t smem = (size_t)(DC_C * (2 * (D + 8) + (END == 1 ? 2 : 1) * DC_LDN) + 2 * D * DC_LDN) * 2;
    static bool attr_set = false;
    if (!attr_set && cudaFuncSetAttribute(decay_chunk_out_kernel<D, NS, END>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
        return kestrel_fail(-3, "decay_chunks: cannot set the shared memory size");
    attr_set = true;
    kestrel_launch(decay_chunk_out_kernel<D, NS, END>, dim3(tiles, p.H), dim3(128), smem, stream, p);
    return kestrel_check_launch("decay_chunk_out");
}

template <int D, int END>
static int dc_out_any(const DecayChunkParams &p, int tiles, cudaStream_t stream) {
    if (p.dv <= 64) return dc_out<D, 1, END>(p, tiles, stream);
    if (p.dv <= 128) return dc_out<D, 2, END>(p, tiles, stream);
    return dc_out<D, 4, END>(p, tiles, stream);
}

KESTREL_API int kestrel_ssm_chunks(const void *act, long long ld_act, const float *step, const float *log_decay, const float *D, const float *partial, int S,
                                   long long slice_stride, int ld, int col_z, float *state, long long state_stride, long long state_off,
                                   const int *cu_seqlens, const int *slots, const int *tile_seq, const int *tile_row0, const int *first_tile, int tiles,
                                   float *scratch, float *y, int nseq, int H, int G, int N, int P, cudaStream_t stream) {
    if (nseq == 0 || tiles == 0) return 0;
    KESTREL_REQUIRE(nseq > 0 && nseq <= 65535 && tiles > 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && N > 0 && P > 0 && N % 8 == 0 && P % 8 == 0 &&
                    N <= 256 && P <= 256, "ssm_chunks: bad sizes H=%d G=%d N=%d P=%d", H, G, N, P);
    KESTREL_REQUIRE(S > 0 && col_z >= 0 && col_z + H * P <= ld && ld % 2 == 0 && col_z % 2 == 0 && slice_stride % 2 == 0 && state_stride % 4 == 0 &&
                    state_off % 4 == 0 && ld_act % 8 == 0 && (((uintptr_t)state | (uintptr_t)act | (uintptr_t)scratch) & 15) == 0,
                    "ssm_chunks: the gate's columns, the rows or the state's place do not fit");
    DecayChunkParams p = {};
    const __nv_bfloat16 *a = (const __nv_bfloat16 *)act;
    p.v = a; p.k = a + H * P; p.q = a + H * P + G * N; p.ldq = p.ldk = p.ldv = ld_act; p.group = H / G;
    p.log_decay = log_decay; p.step = step; p.cu_seqlens = cu_seqlens; p.slots = slots; p.tile_seq = tile_seq; p.tile_row0 = tile_row0;
    p.first_tile = first_tile; p.state = state; p.state_stride = state_stride; p.state_off = state_off;
    const size_t n = (size_t)tiles * H * N * P;
    p.scratch = scratch; p.before = (__nv_bfloat16 *)(scratch + n); p.total = scratch + 2 * n;
    p.gate = partial; p.gate_slices = S; p.gate_ld = ld; p.gate_col0 = col_z; p.gate_stride = slice_stride;
    p.D = D; p.y = y; p.H = H; p.d = N; p.dv = P;
#define SC_CASE(DD)                                              \
    {                                                            \
        int rc = dc_kv_scan<DD>(p, tiles, nseq, stream);         \
        return rc ? rc : dc_out_any<DD, 0>(p, tiles, stream);    \
    }
    if (N <= 32) SC_CASE(32)
    if (N <= 64) SC_CASE(64)
    if (N <= 128) SC_CASE(128)
    SC_CASE(256)
#undef SC_CASE
}

KESTREL_API int kestrel_delta_chunks_out(const void *act, long long ld_act, int G, const void *u_hi, const void *u_lo, const float *q_scale, const float *k_scale,
                                         const float *log_decay, const void *before, const float *w, float eps, const float *partial, int S,
                                         long long slice_stride, int ld, int col_g, const int *cu_seqlens, const int *tile_seq, const int *tile_row0, int tiles,
                                         void *out, int H, int d, int dv, cudaStream_t stream) {
    if (tiles == 0) return 0;
    KESTREL_REQUIRE(tiles > 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && d > 0 && dv > 0 && d % 8 == 0 && dv % 8 == 0 && d <= 128 && dv <= 256,
                    "delta_chunks_out: bad sizes H=%d G=%d d=%d dv=%d", H, G, d, dv);
    KESTREL_REQUIRE(S > 0 && col_g >= 0 && col_g + H * dv <= ld && ld % 2 == 0 && col_g % 2 == 0 && slice_stride % 2 == 0 && ld_act % 8 == 0,
                    "delta_chunks_out: the gate's columns or the rows do not fit");
    DecayChunkParams p = {};
    p.q = (const __nv_bfloat16 *)act; p.k = p.q + G * d; p.v = (const __nv_bfloat16 *)u_hi; p.v_lo = (const __nv_bfloat16 *)u_lo;
    p.ldq = p.ldk = ld_act; p.ldv = (long long)H * dv; p.group = H / G; p.q_scale = q_scale; p.k_scale = k_scale; p.log_decay = log_decay;
    p.cu_seqlens = cu_seqlens; p.tile_seq = tile_seq; p.tile_row0 = tile_row0; p.before = (__nv_bfloat16 *)before;
    p.gate = partial; p.gate_slices = S; p.gate_ld = ld; p.gate_col0 = col_g; p.gate_stride = slice_stride;
    p.w = w; p.eps = eps; p.out = (__nv_bfloat16 *)out; p.H = H; p.d = d; p.dv = dv;
    if (d <= 32) return dc_out_any<32, 1>(p, tiles, stream);
    if (d <= 64) return dc_out_any<64, 1>(p, tiles, stream);
    return dc_out_any<128, 1>(p, tiles, stream);
}
