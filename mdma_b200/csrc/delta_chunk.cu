// The gated delta rule with a decay per key channel, a chunk of sixteen rows at a time (the serving engine's portions of
// prompts).  With L_i[d] the running sum of log decays within the chunk, all rows of a chunk follow from the state S at
// its start without walking them:
//     A_ij = sum_d k_i[d] k_j[d] e^(L_i[d] - L_j[d])  (j < i),      B_ij = sum_d q_i[d] k_j[d] e^(L_i[d] - L_j[d])  (j <= i),
//     u_i  = b_i (v_i - S^T (e^(L_i) k_i) - sum_(j<i) A_ij u_j),    o_i  = S^T (e^(L_i) q_i) + sum_(j<=i) B_ij u_j,
//     S   <- diag(e^(L_n)) S + sum_j (e^(L_n - L_j) k_j) u_j^T.
// No exponent is ever above zero.
//
// delta_chunk_prepare, block = (chunk, head), all chunks side by side: everything that does not depend on S, left in
// scratch as one run of floats per (chunk, head), laid out as the walk's shared memory (`DcLayout`).  It starts from the
// projections: the short convolutions with silu, unit vectors, step sizes and the decays' logarithms are made here too.  The
// triangular system is solved for its two right sides, w_i = b_i (e^(L_i) k_i - sum A_ij w_j) and z_i = b_i (v_i - sum
// A_ij z_j), so that u = z - S^T w; also e^(L_i) q_i, e^(L_n - L_j) k_j, B and e^(L_n).
// delta_chunk_walk, block = (sequence, head, sixteen columns of S), 4 warps, chunks in order: S^T lies in the accumulators
// of mma.sync m16n8k8 (a warp has a quarter of the key channels), which are the left operand of S^T w and S^T q as they
// are; the warps' partial sums meet in shared memory once a chunk.  Products in float precision from tf32 pairs: every
// number is split into the part the tensor core reads and the rest, and three of the four products are summed.
// The next chunks' rows are on their way (cp.async) while a chunk is computed.
#include "delta_rule.cuh"

namespace mdma {

constexpr int kDc = 16;                   // rows of a chunk
constexpr int kDcMaxDim = 256, kDcCols = 16;
constexpr float kDcLog2e = 1.4426950408889634f;

// One (chunk, head) in scratch: w, qg [16][dimP + 8], kd [16][dimP + 4], B [16][24], the whole decay [dimP], then z for every
// sixteen columns [16][20].  dimP: the channels rounded up to a multiple of 32, zero beyond dim; rows beyond the chunk's zero.
struct DcLayout {
    int dimP, wp, kp, qg, kd, b, g, z, slices, floats;
    __host__ __device__ DcLayout(int dim, int vdim) {
        dimP = (dim + 31) / 32 * 32;
        if (dimP > 128) dimP = 256;                       // the sizes the walk is compiled for
        wp = dimP + 8; kp = dimP + 4;
        qg = kDc * wp; kd = 2 * kDc * wp; b = kd + kDc * kp; g = b + kDc * 24; z = g + dimP;
        slices = (vdim + kDcCols - 1) / kDcCols;
        floats = z + slices * kDc * 20;
    }
};
// chunk c of sequence s: chunks of different sequences never share a place
__device__ __forceinline__ size_t dc_place(int seq_start, int s, int chunk) { return (size_t)(seq_start / kDc) + s + chunk; }

__device__ __forceinline__ float dc_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float4 dc_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void dc_st4(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }

// ---------------------------------------------------------------- what does not depend on S
constexpr int kDcTiles = 36, kDcSlices = 7;          // 2 x 2 tiles on and below the diagonal; parts of the channels
static size_t dc_prepare_smem(int dim, int vdim) {
    return sizeof(float) * ((size_t)3 * kDc * (dim + 4) + (size_t)kDc * vdim + 2 * kDc * (kDc + 4) + (size_t)kDcSlices * kDcTiles * 8 + kDc);
}

template <int TAPS>      // the convolution's taps (shorter ones: zeros in front), or 0: any number, every input read again
__global__ void __launch_bounds__(256, 2)
delta_chunk_prepare_kernel(const float* __restrict__ proj, int proj_stride, const float* __restrict__ raw, const void* __restrict__ conv_w,
                           int conv_dtype, int taps, const void* __restrict__ a_log, const void* __restrict__ dt_bias, int vec_dtype,
                           const float* __restrict__ conv_state, size_t state_stride, float* __restrict__ scratch,
                           const int* __restrict__ seq_start, const int* __restrict__ seq_slot, int heads, int kv_heads, int dim,
                           int vdim, int max_chunks, float unit_eps, float q_scale) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float dc_sm[];
    const int s = blockIdx.x / max_chunks, chunk = blockIdx.x - s * max_chunks, h = blockIdx.y;
    const int start = seq_start[s], t0 = start + chunk * kDc;
    const int n = min(kDc, seq_start[s + 1] - t0);
    if (n <= 0) return;
    const DcLayout lay(dim, vdim);
    float* dst = scratch + (dc_place(start, s, chunk) * heads + h) * lay.floats;
    const int hk = h / (heads / kv_heads), P = dim + 4, ap = kDc + 4, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* sk = dc_sm;                        // [16][dim + 4]
    float* sq = sk + kDc * P;
    float* sL = sq + kDc * P;                 // running sums of log2 decays
    float* sv = sL + kDc * P;                 // [16][vdim]
    float* sA = sv + kDc * vdim;              // [16][20]
    float* sB = sA + kDc * ap;
    float* red = sB + kDc * ap;               // [slices][tiles][8]
    float* sb = red + kDcSlices * kDcTiles * 8;
    // convolutions with silu, a thread a channel: q's, k's and v's of this head
    const int qk = kv_heads * dim, channels = 2 * qk + heads * vdim;
    const float* kept = conv_state + (size_t)seq_slot[s] * state_stride;
    for (int e = threadIdx.x; e < 2 * dim + vdim; e += 256) {
        const int ch = e < dim ? hk * dim + e : e < 2 * dim ? qk + hk * dim + e - dim : 2 * qk + h * vdim + e - 2 * dim;
        float* to = e < dim ? sq + e : e < 2 * dim ? sk + e - dim : sv + e - 2 * dim;
        const int pitch = e < 2 * dim ? P : vdim;
        const float* src = proj + (size_t)t0 * proj_stride + ch;
        if (TAPS > 0) {
            float w[TAPS > 0 ? TAPS : 1], x[kDc + (TAPS > 0 ? TAPS : 1) - 1];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j] = j >= TAPS - taps ? delta_weight(conv_w, conv_dtype, (size_t)ch * taps + j - (TAPS - taps)) : 0.f;
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) {
                const int back = TAPS - 1 - j, at = t0 - back - start;           // rows before this step's first: kept inputs
                x[j] = back > taps - 1 ? 0.f : at >= 0 ? src[-(ptrdiff_t)back * proj_stride] : kept[(size_t)(taps - 1 + at) * channels + ch];
            }
#pragma unroll
            for (int i = 0; i < kDc; ++i) x[TAPS - 1 + i] = i < n ? src[(size_t)i * proj_stride] : 0.f;
#pragma unroll
            for (int i = 0; i < kDc; ++i) {
                float acc = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j], x[i + j], acc);
                to[i * pitch] = i < n ? delta_silu(acc) : 0.f;
            }
        } else {
            for (int i = 0; i < kDc; ++i)
                to[i * pitch] = i < n ? delta_conv(proj, proj_stride, kept, conv_w, conv_dtype, taps, channels, t0 + i, start, ch) : 0.f;
        }
    }
    const float rate = -expf(delta_weight(a_log, vec_dtype, h)) * kDcLog2e;
    for (int d = threadIdx.x; d < dim; d += 256) {
        const float bias = delta_weight(dt_bias, vec_dtype, (size_t)h * dim + d);
        const float* src = raw + ((size_t)t0 * heads + h) * dim + d;
        float x[kDc], acc = 0.f;
#pragma unroll
        for (int i = 0; i < kDc; ++i) x[i] = i < n ? src[(size_t)i * heads * dim] : 0.f;
#pragma unroll
        for (int i = 0; i < kDc; ++i) {
            if (i < n) acc = fmaf(rate, delta_softplus(x[i] + bias), acc);
            sL[i * P + d] = acc;
        }
    }
    if (threadIdx.x < kDc) sb[threadIdx.x] = threadIdx.x < n ? delta_sigmoid(proj[(size_t)(t0 + threadIdx.x) * proj_stride + channels + h]) : 0.f;
    for (int e = threadIdx.x; e < 2 * kDc * ap; e += 256) sA[e] = 0.f;              // A, then B
    __syncthreads();
#pragma unroll
    for (int it = 0; it < kDc / 4; ++it) {    // unit vectors, a warp a row of q or k
        float* row = (it & 1 ? sk : sq) + (warp + 8 * (it >> 1)) * P;
        float4 x[2];
        float acc = 0.f;
#pragma unroll
        for (int p = 0; p < 2; ++p) {
            x[p] = 4 * lane + 128 * p < dim ? dc_ld4(row + 4 * lane + 128 * p) : make_float4(0.f, 0.f, 0.f, 0.f);
            acc = fmaf(x[p].x, x[p].x, fmaf(x[p].y, x[p].y, fmaf(x[p].z, x[p].z, fmaf(x[p].w, x[p].w, acc))));
        }
        const float f = (it & 1 ? 1.0f : q_scale) / sqrtf(warp_sum(acc) + unit_eps);
#pragma unroll
        for (int p = 0; p < 2; ++p)
            if (4 * lane + 128 * p < dim) dc_st4(row + 4 * lane + 128 * p, x[p].x * f, x[p].y * f, x[p].z * f, x[p].w * f);
    }
    __syncthreads();
    if (threadIdx.x < kDcTiles * kDcSlices) {
        const int slice = threadIdx.x / kDcTiles, tile = threadIdx.x - slice * kDcTiles;
        int ti = 0;
        while ((ti + 1) * (ti + 2) / 2 <= tile) ++ti;
        const int tj = tile - ti * (ti + 1) / 2;
        const float *k0 = sk + 2 * ti * P, *q0 = sq + 2 * ti * P, *L0 = sL + 2 * ti * P, *x0 = sk + 2 * tj * P, *M0 = sL + 2 * tj * P;
        float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
        // pairs (i, j): (0,0) (0,1) (1,0) (1,1) of the tile; above the diagonal the exponent could be positive: cut off at zero
#define MDMA_DC_PAIRS(c)                                                                                                     \
        {                                                                                                                    \
            const float e00 = xa.c * dc_exp2(l0.c - m0.c), e01 = xb.c * dc_exp2(fminf(l0.c - m1.c, 0.f));                      \
            const float e10 = xa.c * dc_exp2(l1.c - m0.c), e11 = xb.c * dc_exp2(l1.c - m1.c);                                 \
            a[0] = fmaf(ka.c, e00, a[0]); a[1] = fmaf(ka.c, e01, a[1]); a[2] = fmaf(kb.c, e10, a[2]); a[3] = fmaf(kb.c, e11, a[3]); \
            b[0] = fmaf(qa.c, e00, b[0]); b[1] = fmaf(qa.c, e01, b[1]); b[2] = fmaf(qb.c, e10, b[2]); b[3] = fmaf(qb.c, e11, b[3]); \
        }
        for (int d = 4 * slice; d < dim; d += 4 * kDcSlices) {
            const float4 l0 = dc_ld4(L0 + d), l1 = dc_ld4(L0 + P + d), m0 = dc_ld4(M0 + d), m1 = dc_ld4(M0 + P + d);
            const float4 xa = dc_ld4(x0 + d), xb = dc_ld4(x0 + P + d);
            const float4 ka = dc_ld4(k0 + d), kb = dc_ld4(k0 + P + d), qa = dc_ld4(q0 + d), qb = dc_ld4(q0 + P + d);
            MDMA_DC_PAIRS(x) MDMA_DC_PAIRS(y) MDMA_DC_PAIRS(z) MDMA_DC_PAIRS(w)
        }
#undef MDMA_DC_PAIRS
        float* r = red + (slice * kDcTiles + tile) * 8;
        dc_st4(r, a[0], a[1], a[2], a[3]);
        dc_st4(r + 4, b[0], b[1], b[2], b[3]);
    }
    __syncthreads();
    for (int e = threadIdx.x; e < kDcTiles * 8; e += 256) {
        const int tile = e >> 3, x = e & 7;
        int ti = 0;
        while ((ti + 1) * (ti + 2) / 2 <= tile) ++ti;
        const int tj = tile - ti * (ti + 1) / 2, i = 2 * ti + ((x >> 1) & 1), j = 2 * tj + (x & 1);
        float sum = 0.f;
#pragma unroll
        for (int p = 0; p < kDcSlices; ++p) sum += red[(p * kDcTiles + tile) * 8 + x];
        if (x < 4) { if (j < i) sA[i * ap + j] = sum; }
        else if (j <= i) sB[i * ap + j] = sum;
    }
    __syncthreads();
    // the triangular system: a thread per column of w (key channels) and z (value columns)
    const int zcols = lay.slices * kDcCols;
    for (int c = threadIdx.x; c < lay.dimP + zcols; c += 256) {
        const bool key = c < lay.dimP;
        const int cv = c - lay.dimP;
        const bool real = key ? c < dim : cv < vdim;
        float u[kDc];
#pragma unroll
        for (int i = 0; i < kDc; ++i) {
            float r = 0.f;
            if (real) r = key ? sk[i * P + c] * dc_exp2(sL[i * P + c]) : sv[i * vdim + cv];
#pragma unroll
            for (int j4 = 0; j4 < i; j4 += 4) {
                const float4 a4 = dc_ld4(sA + i * ap + j4);      // zero from the diagonal on
                r = fmaf(-a4.x, u[j4], r);
                if (j4 + 1 < i) r = fmaf(-a4.y, u[j4 + 1], r);
                if (j4 + 2 < i) r = fmaf(-a4.z, u[j4 + 2], r);
                if (j4 + 3 < i) r = fmaf(-a4.w, u[j4 + 3], r);
            }
            u[i] = sb[i] * r;
        }
        float* to = key ? dst + c : dst + lay.z + (cv >> 4) * (kDc * 20) + (cv & 15);
        const int pitch = key ? lay.wp : 20;
#pragma unroll
        for (int i = 0; i < kDc; ++i) to[i * pitch] = u[i];
    }
    const float* last = sL + (n - 1) * P;
#pragma unroll
    for (int it = 0; it < kDc / 8; ++it) {
        const int i = warp + 8 * it;
        for (int d = 4 * lane; d < lay.dimP; d += 128) {
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
            if (d < dim && i < n) {
                const float4 L = dc_ld4(sL + i * P + d), E = dc_ld4(last + d), x = dc_ld4(sq + i * P + d), y = dc_ld4(sk + i * P + d);
                a = make_float4(x.x * dc_exp2(L.x), x.y * dc_exp2(L.y), x.z * dc_exp2(L.z), x.w * dc_exp2(L.w));
                b = make_float4(y.x * dc_exp2(E.x - L.x), y.y * dc_exp2(E.y - L.y), y.z * dc_exp2(E.z - L.z), y.w * dc_exp2(E.w - L.w));
            }
            *reinterpret_cast<float4*>(dst + lay.qg + i * lay.wp + d) = a;
            *reinterpret_cast<float4*>(dst + lay.kd + i * lay.kp + d) = b;
        }
    }
    for (int d = threadIdx.x; d < lay.dimP; d += 256) dst[lay.g + d] = d < dim ? dc_exp2(last[d]) : 0.f;
    dst[lay.b + (threadIdx.x >> 4) * 24 + (threadIdx.x & 15)] = sB[(threadIdx.x >> 4) * ap + (threadIdx.x & 15)];
}

// ---------------------------------------------------------------- the walk
constexpr int kDwWarps = 4, kDwStages = 3;

__device__ __forceinline__ void dw_mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// x = hi + lo exactly: hi the bits a tf32 operand keeps, lo the rest (read as tf32 itself)
__device__ __forceinline__ void dw_split(float x, uint32_t& hi, uint32_t& lo) {
    hi = __float_as_uint(x) & 0xffffe000u;
    lo = __float_as_uint(x - __uint_as_float(hi));
}
__device__ __forceinline__ void dw_copy16(void* dst_shared, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"((uint32_t)__cvta_generic_to_shared(dst_shared)), "l"(src) : "memory");
}

// floats of one staged chunk: everything of a (chunk, head) up to z, and z of the block's columns
static __host__ __device__ constexpr int dw_stage_floats(int dimP) { return kDc * (3 * dimP + 20 + 24) + dimP + kDc * 20; }
static size_t dw_smem(int dimP) { return sizeof(float) * ((size_t)kDwStages * dw_stage_floats(dimP) + kDwWarps * 16 * 32); }

// NTD: tiles of eight key channels a warp has (dim up to 32 * NTD)
template <int NTD>
__global__ void __launch_bounds__(kDwWarps * 32)
delta_chunk_walk_kernel(const float* __restrict__ scratch, const int* __restrict__ seq_start, const int* __restrict__ seq_slot,
                        float* __restrict__ state, size_t state_stride, float* __restrict__ out, int heads, int dim, int vdim) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float dw_sm[];
    constexpr int dimP = 32 * NTD, wp = dimP + 8, kp = dimP + 4, zp = 20, bp = 24, stage_floats = dw_stage_floats(dimP);
    constexpr int common = stage_floats - kDc * zp;
    const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kDcCols, cw = min(kDcCols, vdim - c0);
    const int t0 = seq_start[s], t1 = seq_start[s + 1];
    if (t1 <= t0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lr = lane >> 2, lc = lane & 3;
    float* red = dw_sm + (size_t)kDwStages * stage_floats;       // [warp][16][32 lanes]
    const int chunks = (t1 - t0 + kDc - 1) / kDc;
    const DcLayout lay(dim, vdim);
    float* st = state + (size_t)seq_slot[s] * state_stride + (size_t)h * dim * vdim;
    float S[NTD][4];                  // S^T: columns lr, lr + 8; channels warp * 8 NTD + 8 nt + 2 lc, + 1
#pragma unroll
    for (int nt = 0; nt < NTD; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = lr + (e >> 1) * 8, d = warp * 8 * NTD + nt * 8 + 2 * lc + (e & 1);
            S[nt][e] = (c < cw && d < dim) ? st[(size_t)d * vdim + c0 + c] : 0.f;
        }
    const size_t chunk_pitch = (size_t)heads * lay.floats;
    const float* next = scratch + (dc_place(t0, s, 0) * heads + h) * lay.floats + 4 * threadIdx.x;
    const int z_from = lay.z + (int)blockIdx.z * kDc * zp - common;        // the block's z, seen from where `common` ends
    int fill = 0;                                                           // the stage that is filled next
    auto issue = [&](int chunk) {
        if (chunk < chunks) {
            float* to = dw_sm + fill * stage_floats + 4 * threadIdx.x;
#pragma unroll
            for (int e = 0; e < common; e += 4 * kDwWarps * 32)
                if (e + 4 * (int)threadIdx.x < common) dw_copy16(to + e, next + e);
            if (threadIdx.x < kDc * zp / 4) dw_copy16(to + common, next + common + z_from);
            next += chunk_pitch;
            fill = fill + 1 == kDwStages ? 0 : fill + 1;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int p = 0; p < kDwStages - 1; ++p) issue(p);
    int stage = 0;
    float* orow = out + ((size_t)(t0 + (warp & 1) * 8 + 2 * lc) * heads + h) * vdim + c0 + lr;       // warps 0 and 1
    const size_t opitch = (size_t)heads * vdim;
    for (int chunk = 0; chunk < chunks; ++chunk) {
        asm volatile("cp.async.wait_group %0;" :: "n"(kDwStages - 2) : "memory");
        __syncthreads();                       // this chunk is there for everyone; the one before is done with
        issue(chunk + kDwStages - 1);
        const float* sw = dw_sm + stage * stage_floats;
        const float* sqg = sw + kDc * wp;
        const float* skd = sqg + kDc * wp;
        const float* sB = skd + kDc * kp;
        const float* sg = sB + kDc * bp;
        const float* sz = sg + dimP;
        stage = stage + 1 == kDwStages ? 0 : stage + 1;
        // this warp's channels of S^T w and S^T q: [matrix][rows 0-7 | 8-15][4]; the three partial products on their own
        float pa[2][2][4], pb[2][2][4];
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int r = 0; r < 2; ++r)
#pragma unroll
                for (int e = 0; e < 4; ++e) { pa[m][r][e] = 0.f; pb[m][r][e] = 0.f; }
#pragma unroll
        for (int nt = 0; nt < NTD; ++nt) {
            uint32_t ah[4], al[4];            // slots k = lc and lc + 4 are channels 2 lc and 2 lc + 1
            dw_split(S[nt][0], ah[0], al[0]); dw_split(S[nt][2], ah[1], al[1]);
            dw_split(S[nt][1], ah[2], al[2]); dw_split(S[nt][3], ah[3], al[3]);
            const int d = warp * 8 * NTD + nt * 8 + 2 * lc;
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    const float2 x = *reinterpret_cast<const float2*>((m ? sqg : sw) + (r * 8 + lr) * wp + d);
                    uint32_t bh0, bl0, bh1, bl1;
                    dw_split(x.x, bh0, bl0);
                    dw_split(x.y, bh1, bl1);
                    dw_mma(pb[m][r], al[0], al[1], al[2], al[3], bh0, bh1);
                    dw_mma(pb[m][r], ah[0], ah[1], ah[2], ah[3], bl0, bl1);
                    dw_mma(pa[m][r], ah[0], ah[1], ah[2], ah[3], bh0, bh1);
                }
        }
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int r = 0; r < 2; ++r)
                *reinterpret_cast<float4*>(red + ((size_t)(warp * 4 + m * 2 + r) * 32 + lane) * 4) =
                    make_float4(pa[m][r][0] + pb[m][r][0], pa[m][r][1] + pb[m][r][1], pa[m][r][2] + pb[m][r][2], pa[m][r][3] + pb[m][r][3]);
        __syncthreads();
        // u^T = z^T - S^T w, columns lr, lr + 8; rows 8 r + 2 lc, + 1 (every warp has all of it)
        uint32_t uh[2][4], ul[2][4];          // as the left operand: slots of rows 2 lc, 2 lc + 1
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int p = 0; p < kDwWarps; ++p) {
                const float4 x = *reinterpret_cast<const float4*>(red + ((size_t)(p * 4 + r) * 32 + lane) * 4);
                sum.x += x.x; sum.y += x.y; sum.z += x.z; sum.w += x.w;
            }
            const float* zr = sz + (r * 8 + 2 * lc) * zp + lr;
            dw_split(zr[0] - sum.x, uh[r][0], ul[r][0]);
            dw_split(zr[8] - sum.z, uh[r][1], ul[r][1]);
            dw_split(zr[zp] - sum.y, uh[r][2], ul[r][2]);
            dw_split(zr[zp + 8] - sum.w, uh[r][3], ul[r][3]);
        }
        if (warp < 2) {                       // o^T of rows 8 warp .. 8 warp + 7
            float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int p = 0; p < kDwWarps; ++p) {
                const float4 x = *reinterpret_cast<const float4*>(red + ((size_t)(p * 4 + 2 + warp) * 32 + lane) * 4);
                o[0] += x.x; o[1] += x.y; o[2] += x.z; o[3] += x.w;
            }
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const float2 x = *reinterpret_cast<const float2*>(sB + (warp * 8 + lr) * bp + r * 8 + 2 * lc);
                uint32_t bh0, bl0, bh1, bl1;
                dw_split(x.x, bh0, bl0);
                dw_split(x.y, bh1, bl1);
                dw_mma(o, ul[r][0], ul[r][1], ul[r][2], ul[r][3], bh0, bh1);
                dw_mma(o, uh[r][0], uh[r][1], uh[r][2], uh[r][3], bl0, bl1);
                dw_mma(o, uh[r][0], uh[r][1], uh[r][2], uh[r][3], bh0, bh1);
            }
            const int left = t1 - t0 - chunk * kDc - warp * 8 - 2 * lc;
            if (lr < cw) {
                if (left > 0) orow[0] = o[0];
                if (left > 1) orow[opitch] = o[1];
            }
            if (lr + 8 < cw) {
                if (left > 0) orow[8] = o[2];
                if (left > 1) orow[opitch + 8] = o[3];
            }
            orow += kDc * opitch;
        }
        // S^T <- S^T e^(L_n) + u^T kd
#pragma unroll
        for (int nt = 0; nt < NTD; ++nt) {
            const int d = warp * 8 * NTD + nt * 8;
            const float2 g = *reinterpret_cast<const float2*>(sg + d + 2 * lc);
            float big[4] = {S[nt][0] * g.x, S[nt][1] * g.y, S[nt][2] * g.x, S[nt][3] * g.y}, small[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const float* kr = skd + (r * 8 + 2 * lc) * kp + d + lr;
                uint32_t bh0, bl0, bh1, bl1;
                dw_split(kr[0], bh0, bl0);
                dw_split(kr[kp], bh1, bl1);
                dw_mma(small, ul[r][0], ul[r][1], ul[r][2], ul[r][3], bh0, bh1);
                dw_mma(small, uh[r][0], uh[r][1], uh[r][2], uh[r][3], bl0, bl1);
                dw_mma(big, uh[r][0], uh[r][1], uh[r][2], uh[r][3], bh0, bh1);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) S[nt][e] = big[e] + small[e];
        }
    }
#pragma unroll
    for (int nt = 0; nt < NTD; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = lr + (e >> 1) * 8, d = warp * 8 * NTD + nt * 8 + 2 * lc + (e & 1);
            if (c < cw && d < dim) st[(size_t)d * vdim + c0 + c] = S[nt][e];
        }
}

}  // namespace mdma

using namespace mdma;

extern "C" {

// Floats of scratch a step of n_rows rows in n_seqs sequences needs.
long mdma_delta_chunks_scratch(int n_rows, int n_seqs, int heads, int dim, int vdim) {
    return ((long)n_rows / kDc + n_seqs + 1) * heads * (long)DcLayout(dim, vdim).floats;
}

// proj rows [q | k | v | b | ..], raw [rows][heads * dim] the decays' inputs, out [rows][heads * vdim], all floats; the
// convolutions' kept inputs are read, not brought up to date
int mdma_delta_chunks(const float* proj, int proj_stride, const float* raw, const void* conv_w, int conv_dtype, int taps,
                      const void* a_log, const void* dt_bias, int vec_dtype, const float* conv_state, float* scratch,
                      long scratch_floats, const int* seq_start, const int* seq_slot, float* state, long state_stride, float* out,
                      int n_rows, int n_seqs, int max_new, int heads, int kv_heads, int dim, int vdim, float unit_eps,
                      float q_scale, cudaStream_t stream) {
    MDMA_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0, "delta_chunks: bad sizes");
    MDMA_REQUIRE(dim <= kDcMaxDim && dim % 4 == 0 && vdim % 4 == 0 && vdim <= 512, "delta_chunks: heads of %d x %d are not a geometry this kernel takes", dim, vdim);
    MDMA_REQUIRE(taps >= 1 && taps <= kDeltaMaxTaps, "delta_chunks: %d taps, the kernel takes 1..%d", taps, kDeltaMaxTaps);
    MDMA_REQUIRE(((uintptr_t)scratch & 15) == 0, "delta_chunks: scratch must start on 16 bytes");
    if (n_rows == 0 || n_seqs == 0) return 0;
    const long need = mdma_delta_chunks_scratch(n_rows, n_seqs, heads, dim, vdim);
    MDMA_REQUIRE(scratch_floats >= need, "delta_chunks: %ld floats of scratch needed, %ld given", need, scratch_floats);
    const int max_chunks = (max_new + kDc - 1) / kDc;
    MDMA_REQUIRE((long)n_seqs * max_chunks <= 2147483647l && heads <= 65535, "delta_chunks: too many rows");
#define MDMA_DC_PREPARE(TAPS)                                                                                               \
    do {                                                                                                                   \
        static bool raised = false;                                                                                        \
        if (!raised) { cudaFuncSetAttribute(delta_chunk_prepare_kernel<TAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 120 * 1024); raised = true; } \
        launch_chained(delta_chunk_prepare_kernel<TAPS>, dim3((unsigned)(n_seqs * max_chunks), heads), dim3(256),          \
                       dc_prepare_smem(dim, vdim), stream, proj, proj_stride, raw, conv_w, conv_dtype, taps, a_log, dt_bias, \
                       vec_dtype, conv_state, (size_t)state_stride, scratch, seq_start, seq_slot, heads, kv_heads, dim, vdim, \
                       max_chunks, unit_eps, q_scale);                                                                     \
    } while (0)
    if (taps <= 4) MDMA_DC_PREPARE(4); else MDMA_DC_PREPARE(0);
#undef MDMA_DC_PREPARE
    MDMA_LAUNCH_OK("delta_chunk_prepare");
    const DcLayout lay(dim, vdim);
    dim3 grid(n_seqs, heads, lay.slices);
#define MDMA_DW(NTD)                                                                                                     \
    do {                                                                                                                 \
        static bool up = false;                                                                                          \
        if (!up) { cudaFuncSetAttribute(delta_chunk_walk_kernel<NTD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)dw_smem(32 * NTD)); up = true; } \
        launch_chained(delta_chunk_walk_kernel<NTD>, grid, dim3(kDwWarps * 32), dw_smem(32 * NTD), stream, (const float*)scratch, \
                       seq_start, seq_slot, state, (size_t)state_stride, out, heads, dim, vdim);                         \
    } while (0)
    if (lay.dimP == 32) MDMA_DW(1);
    else if (lay.dimP == 64) MDMA_DW(2);
    else if (lay.dimP == 96) MDMA_DW(3);
    else if (lay.dimP == 128) MDMA_DW(4);
    else MDMA_DW(8);
#undef MDMA_DW
    MDMA_LAUNCH_OK("delta_chunk_walk");
    return 0;
}

}  // extern "C"
