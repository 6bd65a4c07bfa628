// The gated delta rule with a decay per key channel, a chunk of sixteen rows at a time (the serving engine's portions of
// prompts).  With L_i[d] the running sum of log decays within the chunk, all rows of a chunk follow from the state S at
// its start without walking them:
//     A_ij = sum_d k_i[d] k_j[d] e^(L_i[d] - L_j[d])  (j < i),      B_ij = sum_d q_i[d] k_j[d] e^(L_i[d] - L_j[d])  (j <= i),
//     u_i  = b_i (v_i - S^T (e^(L_i) k_i) - sum_(j<i) A_ij u_j),    o_i  = S^T (e^(L_i) q_i) + sum_(j<=i) B_ij u_j,
//     S   <- diag(e^(L_n)) S + sum_j (e^(L_n - L_j) k_j) u_j^T.
// No exponent is ever above zero.
//
// delta_chunk_prepare, block = (chunk, head), all chunks side by side: everything that does not depend on S.  The
// triangular system is solved for its two right sides, w_i = b_i (e^(L_i) k_i - sum A_ij w_j) and z_i = b_i (v_i - sum
// A_ij z_j), so that u = z - S^T w; also e^(L_i) q_i, e^(L_n - L_j) k_j, B and e^(L_n).
// delta_chunk_walk, block = (sequence, head, sixteen columns of S), 4 warps, chunks in order: S^T lies in the accumulators
// of mma.sync m16n8k8 (a warp has a quarter of the key channels), which are the left operand of S^T w and S^T q as they
// are; the warps' partial sums meet in shared memory once a chunk.  Products in float precision from tf32 pairs: every
// number is split into the part the tensor core reads and the rest, and three of the four products are summed.
// The next chunks' rows are on their way (cp.async) while a chunk is computed.
#include "common.cuh"

namespace mdma {

constexpr int kDc = 16;                   // rows of a chunk
constexpr int kDcMaxDim = 256;
constexpr float kDcLog2e = 1.4426950408889634f;

// ---------------------------------------------------------------- what does not depend on S
constexpr int kDcTiles = 36, kDcSlices = 7;          // 2 x 2 tiles on and below the diagonal; parts of the channels
static size_t dc_prepare_smem(int dim) {
    return sizeof(float) * ((size_t)3 * kDc * (dim + 1) + 2 * kDc * (kDc + 4) + (size_t)kDcSlices * kDcTiles * 8 + kDc);
}

__global__ void __launch_bounds__(256, 2)
delta_chunk_prepare_kernel(const float* __restrict__ q, const float* __restrict__ k, float* __restrict__ v, float* __restrict__ lg,
                           const float* __restrict__ beta, float* __restrict__ w, float* __restrict__ qg, float* __restrict__ kd,
                           float* __restrict__ bm, const int* __restrict__ seq_start, int heads, int kv_heads, int dim, int vdim,
                           int max_chunks) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float dc_sm[];
    const int s = blockIdx.x / max_chunks, h = blockIdx.y;
    const int t0 = seq_start[s] + (int)(blockIdx.x % max_chunks) * kDc;
    const int n = min(kDc, seq_start[s + 1] - t0);
    if (n <= 0) return;
    const int hk = h / (heads / kv_heads), P = dim + 1, ap = kDc + 4;
    float* sk = dc_sm;                        // [16][dim + 1]
    float* sq = sk + kDc * P;
    float* sL = sq + kDc * P;                 // running sums of log2 decays
    float* sA = sL + kDc * P + ((4 - (3 * kDc * P) % 4) & 3);        // [16][20], rows on 16-byte boundaries
    float* sB = sA + kDc * ap;
    float* red = sB + kDc * ap;               // [slices][tiles][8]
    float* sb = red + kDcSlices * kDcTiles * 8;
    for (int e = threadIdx.x; e < kDc * dim; e += blockDim.x) {
        const int i = e / dim, d = e - i * dim;
        const bool have = i < n;
        sk[i * P + d] = have ? k[((size_t)(t0 + i) * kv_heads + hk) * dim + d] : 0.f;
        sq[i * P + d] = have ? q[((size_t)(t0 + i) * kv_heads + hk) * dim + d] : 0.f;
        sL[i * P + d] = have ? lg[((size_t)(t0 + i) * heads + h) * dim + d] * kDcLog2e : 0.f;
    }
    if (threadIdx.x < kDc) sb[threadIdx.x] = threadIdx.x < n ? beta[(size_t)(t0 + threadIdx.x) * heads + h] : 0.f;
    __syncthreads();
    for (int d = threadIdx.x; d < dim; d += blockDim.x) {
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < kDc; ++i) { acc += sL[i * P + d]; sL[i * P + d] = acc; }
    }
    __syncthreads();
    if (threadIdx.x < kDcTiles * kDcSlices) {
        const int tile = threadIdx.x % kDcTiles, slice = threadIdx.x / kDcTiles;
        int ti = 0;
        while ((ti + 1) * (ti + 2) / 2 <= tile) ++ti;
        const int tj = tile - ti * (ti + 1) / 2;
        const float *k0 = sk + 2 * ti * P, *k1 = k0 + P, *q0 = sq + 2 * ti * P, *q1 = q0 + P, *L0 = sL + 2 * ti * P, *L1 = L0 + P;
        const float *x0 = sk + 2 * tj * P, *x1 = x0 + P, *M0 = sL + 2 * tj * P, *M1 = M0 + P;
        float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
        // pairs (i, j): (0,0) (0,1) (1,0) (1,1) of the tile; above the diagonal the exponent could be positive: cut off at zero
        for (int d = slice; d < dim; d += kDcSlices) {
            const float l0 = L0[d], l1 = L1[d], m0 = M0[d], m1 = M1[d];
            const float e00 = x0[d] * exp2f(l0 - m0), e01 = x1[d] * exp2f(fminf(l0 - m1, 0.f));
            const float e10 = x0[d] * exp2f(l1 - m0), e11 = x1[d] * exp2f(l1 - m1);
            const float ka = k0[d], kb = k1[d], qa = q0[d], qb = q1[d];
            a[0] = fmaf(ka, e00, a[0]); a[1] = fmaf(ka, e01, a[1]); a[2] = fmaf(kb, e10, a[2]); a[3] = fmaf(kb, e11, a[3]);
            b[0] = fmaf(qa, e00, b[0]); b[1] = fmaf(qa, e01, b[1]); b[2] = fmaf(qb, e10, b[2]); b[3] = fmaf(qb, e11, b[3]);
        }
        float* r = red + (slice * kDcTiles + tile) * 8;
#pragma unroll
        for (int e = 0; e < 4; ++e) { r[e] = a[e]; r[4 + e] = b[e]; }
    }
    for (int e = threadIdx.x; e < 2 * kDc * ap; e += blockDim.x) sA[e] = 0.f;        // A, then B
    __syncthreads();
    for (int e = threadIdx.x; e < kDcTiles * 8; e += blockDim.x) {
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
    for (int c = threadIdx.x; c < dim + vdim; c += blockDim.x) {
        const bool key = c < dim;
        float u[kDc];
#pragma unroll
        for (int i = 0; i < kDc; ++i) {
            float r = 0.f;
            if (key) r = sk[i * P + c] * exp2f(sL[i * P + c]);
            else if (i < n) r = v[((size_t)(t0 + i) * heads + h) * vdim + c - dim];
#pragma unroll
            for (int j4 = 0; j4 < i; j4 += 4) {
                const float4 a4 = *reinterpret_cast<const float4*>(sA + i * ap + j4);      // zero from the diagonal on
                r = fmaf(-a4.x, u[j4], r);
                if (j4 + 1 < i) r = fmaf(-a4.y, u[j4 + 1], r);
                if (j4 + 2 < i) r = fmaf(-a4.z, u[j4 + 2], r);
                if (j4 + 3 < i) r = fmaf(-a4.w, u[j4 + 3], r);
            }
            u[i] = sb[i] * r;
        }
#pragma unroll
        for (int i = 0; i < kDc; ++i)
            if (i < n) {
                if (key) w[((size_t)(t0 + i) * heads + h) * dim + c] = u[i];
                else v[((size_t)(t0 + i) * heads + h) * vdim + c - dim] = u[i];
            }
    }
    const float* last = sL + (n - 1) * P;
    for (int e = threadIdx.x; e < n * dim; e += blockDim.x) {
        const int i = e / dim, d = e - i * dim;
        const size_t at = ((size_t)(t0 + i) * heads + h) * dim + d;
        qg[at] = sq[i * P + d] * exp2f(sL[i * P + d]);
        kd[at] = sk[i * P + d] * exp2f(last[d] - sL[i * P + d]);
        if (i == 0) lg[at] = exp2f(last[d]);              // the chunk's whole decay takes the place of its first row's
    }
    for (int e = threadIdx.x; e < n * kDc; e += blockDim.x)
        bm[((size_t)(t0 + e / kDc) * heads + h) * kDc + e % kDc] = sB[(e / kDc) * ap + e % kDc];
}

// ---------------------------------------------------------------- the walk
constexpr int kDwCols = 16, kDwWarps = 4, kDwStages = 4;

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

// floats of one staged chunk: w, qg [16][dimP + 8]; kd [16][dimP + 4]; z [16][20]; B [16][24]; whole decay [dimP]
static __host__ __device__ int dw_stage_floats(int dimP) { return kDc * (3 * dimP + 20 + 20 + 24) + dimP; }
static size_t dw_smem(int dimP) { return sizeof(float) * ((size_t)kDwStages * dw_stage_floats(dimP) + kDwWarps * 16 * 32); }

// NTD: tiles of eight key channels a warp has (dim up to 32 * NTD)
template <int NTD>
__global__ void __launch_bounds__(kDwWarps * 32)
delta_chunk_walk_kernel(const float* __restrict__ w, const float* __restrict__ qg, const float* __restrict__ kd,
                        const float* __restrict__ z, const float* __restrict__ bm, const float* __restrict__ whole,
                        const int* __restrict__ seq_start, const int* __restrict__ seq_slot, float* __restrict__ state,
                        size_t state_stride, float* __restrict__ out, int heads, int dim, int vdim) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float dw_sm[];
    constexpr int dimP = 32 * NTD, wp = dimP + 8, kp = dimP + 4, zp = 20, bp = 24;
    const int s = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * kDwCols, cw = min(kDwCols, vdim - c0);
    const int t0 = seq_start[s], t1 = seq_start[s + 1];
    if (t1 <= t0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lr = lane >> 2, lc = lane & 3;
    const int stage_floats = dw_stage_floats(dimP);
    float* red = dw_sm + (size_t)kDwStages * stage_floats;       // [warp][16][32 lanes]
    for (int e = threadIdx.x; e < kDwStages * stage_floats; e += blockDim.x) dw_sm[e] = 0.f;      // padding stays zero
    const int chunks = (t1 - t0 + kDc - 1) / kDc, d4 = dim >> 2, c4 = cw >> 2;
    float* st = state + (size_t)seq_slot[s] * state_stride + (size_t)h * dim * vdim;
    float S[NTD][4];                  // S^T: columns lr, lr + 8; channels warp * 8 NTD + 8 nt + 2 lc, + 1
#pragma unroll
    for (int nt = 0; nt < NTD; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int c = lr + (e >> 1) * 8, d = warp * 8 * NTD + nt * 8 + 2 * lc + (e & 1);
            S[nt][e] = (c < cw && d < dim) ? st[(size_t)d * vdim + c0 + c] : 0.f;
        }
    __syncthreads();
    auto issue = [&](int chunk) {
        if (chunk < chunks) {
            float* sw = dw_sm + (size_t)(chunk % kDwStages) * stage_floats;
            float* sqg = sw + kDc * wp;
            float* skd = sqg + kDc * wp;
            float* sz = skd + kDc * kp;
            float* sB = sz + kDc * zp;
            float* sg = sB + kDc * bp;
            const int r0 = t0 + chunk * kDc, n = min(kDc, t1 - r0);
            for (int e = threadIdx.x; e < kDc * d4; e += blockDim.x) {
                const int i = e / d4, p = (e - i * d4) << 2;
                if (i < n) {
                    const size_t at = ((size_t)(r0 + i) * heads + h) * dim + p;
                    dw_copy16(sw + i * wp + p, w + at);
                    dw_copy16(sqg + i * wp + p, qg + at);
                    dw_copy16(skd + i * kp + p, kd + at);
                } else {
                    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
                    *reinterpret_cast<float4*>(sw + i * wp + p) = zero;
                    *reinterpret_cast<float4*>(sqg + i * wp + p) = zero;
                    *reinterpret_cast<float4*>(skd + i * kp + p) = zero;
                }
            }
            for (int e = threadIdx.x; e < kDc * 4; e += blockDim.x) {
                const int i = e >> 2, p = (e & 3) << 2;
                const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i < n) {
                    if ((e & 3) < c4) dw_copy16(sz + i * zp + p, z + ((size_t)(r0 + i) * heads + h) * vdim + c0 + p);
                    dw_copy16(sB + i * bp + p, bm + ((size_t)(r0 + i) * heads + h) * kDc + p);
                } else {
                    *reinterpret_cast<float4*>(sz + i * zp + p) = zero;
                    *reinterpret_cast<float4*>(sB + i * bp + p) = zero;
                }
            }
            for (int e = threadIdx.x; e < d4; e += blockDim.x) dw_copy16(sg + 4 * e, whole + ((size_t)r0 * heads + h) * dim + 4 * e);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int p = 0; p < kDwStages - 1; ++p) issue(p);
    for (int chunk = 0; chunk < chunks; ++chunk) {
        asm volatile("cp.async.wait_group %0;" :: "n"(kDwStages - 2) : "memory");
        __syncthreads();                       // this chunk is there for everyone; the one before is done with
        issue(chunk + kDwStages - 1);
        const float* sw = dw_sm + (size_t)(chunk % kDwStages) * stage_floats;
        const float* sqg = sw + kDc * wp;
        const float* skd = sqg + kDc * wp;
        const float* sz = skd + kDc * kp;
        const float* sB = sz + kDc * zp;
        const float* sg = sB + kDc * bp;
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
            const int i0 = chunk * kDc + warp * 8 + 2 * lc;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int c = lr + (e >> 1) * 8, i = i0 + (e & 1);
                if (c < cw && t0 + i < t1) out[((size_t)(t0 + i) * heads + h) * vdim + c0 + c] = o[e];
            }
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

// q, k [rows][kv_heads * dim], v [rows][heads * vdim] (becomes z), lg [rows][heads * dim] (a chunk's first row becomes its
// whole decay), beta [rows][heads]; w, qg, kd [rows][heads * dim] and bm [rows][heads * 16] are scratch; out [rows][heads * vdim]
int mdma_delta_chunks(const float* q, const float* k, float* v, float* lg, const float* beta, float* w, float* qg, float* kd,
                      float* bm, const int* seq_start, const int* seq_slot, float* state, long state_stride, float* out,
                      int n_rows, int n_seqs, int max_new, int heads, int kv_heads, int dim, int vdim, cudaStream_t stream) {
    MDMA_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0, "delta_chunks: bad sizes");
    MDMA_REQUIRE(dim <= kDcMaxDim && dim % 4 == 0 && vdim % 4 == 0, "delta_chunks: heads of %d x %d are not a geometry this kernel takes", dim, vdim);
    MDMA_REQUIRE((((uintptr_t)v | (uintptr_t)lg | (uintptr_t)w | (uintptr_t)qg | (uintptr_t)kd | (uintptr_t)bm) & 15) == 0, "delta_chunks: rows must start on 16 bytes");
    if (n_rows == 0 || n_seqs == 0) return 0;
    const int max_chunks = (max_new + kDc - 1) / kDc;
    MDMA_REQUIRE((long)n_seqs * max_chunks <= 2147483647l && heads <= 65535, "delta_chunks: too many rows");
    static bool raised = false;
    if (!raised) {
        cudaFuncSetAttribute(delta_chunk_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
        raised = true;
    }
    launch_chained(delta_chunk_prepare_kernel, dim3((unsigned)(n_seqs * max_chunks), heads), dim3(256), dc_prepare_smem(dim) + 16, stream,
                   q, k, v, lg, beta, w, qg, kd, bm, seq_start, heads, kv_heads, dim, vdim, max_chunks);
    MDMA_LAUNCH_OK("delta_chunk_prepare");
    dim3 grid(n_seqs, heads, (vdim + kDwCols - 1) / kDwCols);
#define MDMA_DW(NTD)                                                                                                     \
    do {                                                                                                                 \
        static bool up = false;                                                                                          \
        if (!up) { cudaFuncSetAttribute(delta_chunk_walk_kernel<NTD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)dw_smem(32 * NTD)); up = true; } \
        launch_chained(delta_chunk_walk_kernel<NTD>, grid, dim3(kDwWarps * 32), dw_smem(32 * NTD), stream, (const float*)w,  \
                       (const float*)qg, (const float*)kd, (const float*)v, (const float*)bm, (const float*)lg, seq_start, \
                       seq_slot, state, (size_t)state_stride, out, heads, dim, vdim);                                    \
    } while (0)
    if (dim <= 32) MDMA_DW(1);
    else if (dim <= 64) MDMA_DW(2);
    else if (dim <= 96) MDMA_DW(3);
    else if (dim <= 128) MDMA_DW(4);
    else MDMA_DW(8);
#undef MDMA_DW
    MDMA_LAUNCH_OK("delta_chunk_walk");
    return 0;
}

}  // extern "C"
