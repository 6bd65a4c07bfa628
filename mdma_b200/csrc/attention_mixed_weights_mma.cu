// Attention whose heads' softmax weights are mixed before they meet the values, on the tensor cores (bfloat16,
// mma.sync m16n8k16, float sums).
//
// w'_h = sum_g M[h, g] w_g applied to the values of head h's own kv head c(h) is
//     o_h = sum_g M[h, g] O[g, c(h)],      O[g, c] = sum_j w_g(j) v_c(j),
// so every head g first attends over ALL value heads of a token side by side, as they lie in the cache row (kv_heads *
// v_dim numbers), in one pass with the usual online softmax; the mixing is a small float sum over the finished rows.
//
// Scores: x = factor_g (q_g . k), with a soft cap c: c tanh(x / c), tanh as 1 - 2 / (1 + e^(2 x / c)).  Visible keys are
// numbered without the gap between the first `keep_first` tokens and the window (index e is position e below the gap,
// e + gap above it), so chunks of 32 keys are dense.
//
// mixed_rows (portions of prompts): block = 4 warps, a warp = 16 query rows of one head; the block's heads share a kv
//   head, so a chunk's keys and values are copied once (cp.async, the next chunk on its way while this one is computed).
//   A block takes up to 256 value columns (more: another block computes the scores again).  O goes to scratch in float,
//   `mixed_sum` mixes it.  Long steps run slab by slab of tokens, so that the scratch stays small.
// mixed_step (single tokens): block = (sequence, run of keys), all heads: keys and values of 32 tokens are staged once;
//   scores of a kv head's query heads are one 16-row tile, softmax a warp per head, then all heads as the rows of one
//   product with the value rows.  Unnormalised sums per run of keys; `mixed_merge` adds them in order and mixes.
#include "common.cuh"

namespace mdma {

constexpr int kMwChunk = 32, kMwWarps = 4, kMwTile = 16, kMwStepWarps = 8, kMwMaxHeads = 32;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ void mw_ldmatrix_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mw_ldmatrix_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mw_ldmatrix_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void mw_mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mw_copy16(void* dst_shared, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"((uint32_t)__cvta_generic_to_shared(dst_shared)), "l"(src) : "memory");
}
__device__ __forceinline__ void mw_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void mw_wait() { asm volatile("cp.async.wait_group %0;" :: "n"(N) : "memory"); }
__device__ __forceinline__ uint32_t mw_pack(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float mw_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// a raw dot product as a score in powers of two: `a` = cap log2(e) and `b` = 2 log2(e) factor / cap, or b = log2(e) factor
__device__ __forceinline__ float mw_score(float x, bool capped, float a, float b) {
    return capped ? fmaf(-2.0f * a, __fdividef(1.0f, 1.0f + mw_exp2(x * b)), a) : x * b;
}

struct MwCache {
    const __nv_bfloat16* k;
    const __nv_bfloat16* v;
    const int* pages;        // the sequence's row of the page table
    int page_size, n_kv_heads, dim, v_dim;
    __device__ __forceinline__ size_t row(int p) const { return (size_t)pages[p / page_size] * page_size + (size_t)(p % page_size); }
};

static size_t mw_rows_smem(int dim, int vt) {
    return ((size_t)kMwWarps * kMwTile * (dim + 8) + 2 * (size_t)kMwChunk * ((dim + 8) + (8 * vt + 8))) * 2;
}

// VT: value n-tiles of eight columns a warp accumulates.
// KD: the head size over sixteen where it is known at compile time, else 0.
template <int VT, int KD>
__global__ void __launch_bounds__(kMwWarps * 32, 2)
mixed_rows_kernel(const __nv_bfloat16* __restrict__ q, int q_row_stride, const __nv_bfloat16* __restrict__ k_cache,
                  const __nv_bfloat16* __restrict__ v_cache, const float* __restrict__ factor, float softcap,
                  const int* __restrict__ seq_start, const int* __restrict__ seq_pos0, const int* __restrict__ seq_slot,
                  const int* __restrict__ page_table, int max_pages, int page_size, float* __restrict__ sums, int n_heads,
                  int n_kv_heads, int dim_, int v_dim, int window, int keep_first, int heads_per_block, int cols,
                  int slab0, int slab1) {
    const int dim = KD > 0 ? 16 * KD : dim_;
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) unsigned char mw_smem[];
    const int s = blockIdx.z;
    const int t0 = seq_start[s], n_new = seq_start[s + 1] - t0;
    const int lo_row = max(0, slab0 - t0), hi_row = min(n_new, slab1 - t0);
    const int row_tiles = kMwWarps / heads_per_block, block_rows = row_tiles * kMwTile;
    // the last rows of a prompt see the most keys: they start first
    const int tiles = (max(0, hi_row - lo_row) + block_rows - 1) / block_rows;
    if ((int)blockIdx.x >= tiles) return;
    const int b0 = lo_row + (tiles - 1 - (int)blockIdx.x) * block_rows;
    const int head_blocks = n_heads / heads_per_block;
    const int c0 = ((int)blockIdx.y / head_blocks) * cols, total = n_kv_heads * v_dim, cw = min(cols, total - c0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = ((int)blockIdx.y % head_blocks) * heads_per_block + warp % heads_per_block;
    const int kvh = h / (n_heads / n_kv_heads);
    const int r0 = b0 + (warp / heads_per_block) * kMwTile;
    const int rows = min(kMwTile, hi_row - r0);                            // may be <= 0: the warp only helps with copies
    const int last = seq_pos0[s] + min(b0 + block_rows, hi_row) - 1;       // the block's last position
    const int pos_b = seq_pos0[s] + b0;
    const int first = window > 0 ? max(0, pos_b + 1 - window) : 0;
    const int kept = min(keep_first, first), gap = first - kept, n_keys = last + 1 - gap;
    const MwCache cache = {k_cache, v_cache, page_table + (size_t)seq_slot[s] * max_pages, page_size, n_kv_heads, dim, v_dim};
    constexpr int vp = VT * 8 + 8;
    const int qp = dim + 8;
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(mw_smem) + (size_t)warp * kMwTile * qp;
    __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(mw_smem) + (size_t)kMwWarps * kMwTile * qp;      // [2][32][dim + 8]
    __nv_bfloat16* sv = sk + 2 * (size_t)kMwChunk * qp;                                                    // [2][32][8 VT + 8]
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    for (int e = lane; e < kMwTile * (dim / 8); e += 32) {
        const int r = e / (dim / 8), d8 = e % (dim / 8);
        uint4 v = zero4;
        if (r < rows) v = *reinterpret_cast<const uint4*>(q + (size_t)(t0 + r0 + r) * q_row_stride + (size_t)h * dim + d8 * 8);
        *reinterpret_cast<uint4*>(sq + (size_t)r * qp + d8 * 8) = v;
    }
    auto issue = [&](int e0, int buf) {
        for (int j = warp; j < kMwChunk; j += kMwWarps) {
            __nv_bfloat16* dk = sk + ((size_t)buf * kMwChunk + j) * qp;
            __nv_bfloat16* dv = sv + ((size_t)buf * kMwChunk + j) * vp;
            const int e = e0 + j;
            if (e < n_keys) {
                const size_t row = cache.row(e < kept ? e : e + gap);
                const __nv_bfloat16* gk = k_cache + (row * n_kv_heads + kvh) * dim;
                const __nv_bfloat16* gv = v_cache + row * total + c0;
                for (int d8 = lane; d8 < dim / 8; d8 += 32) mw_copy16(dk + d8 * 8, gk + d8 * 8);
                for (int d8 = lane; d8 < cw / 8; d8 += 32) mw_copy16(dv + d8 * 8, gv + d8 * 8);
            } else {                                                       // rows no key owns: zero
                for (int d8 = lane; d8 < dim / 8; d8 += 32) *reinterpret_cast<uint4*>(dk + d8 * 8) = zero4;
                for (int d8 = lane; d8 < cw / 8; d8 += 32) *reinterpret_cast<uint4*>(dv + d8 * 8) = zero4;
            }
        }
        mw_commit();
    };
    // columns beyond the block's: zero, and computed along with the others
    for (int e = threadIdx.x; e < 2 * kMwChunk * (VT - cw / 8); e += kMwWarps * 32)
        *reinterpret_cast<uint4*>(sv + (size_t)(e / (VT - cw / 8)) * vp + cw + (e % (VT - cw / 8)) * 8) = zero4;
    float o[VT][4];
#pragma unroll
    for (int n = 0; n < VT; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    const int row_lo = lane >> 2, row_hi = row_lo + 8;
    const int w0 = seq_pos0[s] + r0;                                        // position of the warp's first row
    const int p_lo = w0 + row_lo, p_hi = w0 + row_hi;
    const int in_lo = window > 0 ? p_lo + 1 - window : 0, in_hi = window > 0 ? p_hi + 1 - window : 0;
    const bool capped = softcap > 0.f;
    const float ca = softcap * kLog2e, cb = capped ? 2.0f * kLog2e * factor[h] / softcap : kLog2e * factor[h];
    const uint32_t sq_addr = (uint32_t)__cvta_generic_to_shared(sq);
    issue(0, 0);
    for (int e0 = 0, buf = 0; e0 < n_keys; e0 += kMwChunk, buf ^= 1) {
        if (e0 + kMwChunk < n_keys) { issue(e0 + kMwChunk, buf ^ 1); mw_wait<1>(); } else { mw_wait<0>(); }
        __syncthreads();
        const uint32_t sk_addr = (uint32_t)__cvta_generic_to_shared(sk + (size_t)buf * kMwChunk * qp);
        const uint32_t sv_addr = (uint32_t)__cvta_generic_to_shared(sv + (size_t)buf * kMwChunk * vp);
        // whether any of the chunk's keys is visible to any of the warp's rows
        const int p_first = e0 < kept ? e0 : e0 + gap, e_last = min(e0 + kMwChunk, n_keys) - 1, p_last = e_last < kept ? e_last : e_last + gap;
        const bool some = rows > 0 && p_first <= w0 + rows - 1 && (p_first < keep_first || window == 0 || p_last >= w0 + 1 - window);
        if (some) {
            float sc[4][4];
#pragma unroll
            for (int n = 0; n < 4; ++n) { sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f; }
#pragma unroll(KD > 0 ? KD : 4)
            for (int k0 = 0; k0 < dim; k0 += 16) {
                uint32_t a0, a1, a2, a3;
                mw_ldmatrix_x4(sq_addr + (uint32_t)(((lane & 15) * qp + k0 + (lane >> 4) * 8) * 2), a0, a1, a2, a3);
#pragma unroll
                for (int n2 = 0; n2 < 2; ++n2) {
                    uint32_t b0_, b1_, b2_, b3_;
                    const int krow = n2 * 16 + (lane & 7) + (lane >> 4) * 8;
                    mw_ldmatrix_x4(sk_addr + (uint32_t)((krow * qp + k0 + ((lane >> 3) & 1) * 8) * 2), b0_, b1_, b2_, b3_);
                    mw_mma(sc[n2 * 2], a0, a1, a2, a3, b0_, b1_);
                    mw_mma(sc[n2 * 2 + 1], a0, a1, a2, a3, b2_, b3_);
                }
            }
            // every key of the chunk visible to every row of the warp: no mask
            const bool plain = p_last <= w0 && e_last == e0 + kMwChunk - 1 && (window == 0 || p_first >= w0 + kMwTile - window || p_last < keep_first);
            float c_lo = -INFINITY, c_hi = -INFINITY;
#pragma unroll
            for (int n = 0; n < 4; ++n) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    sc[n][i] = mw_score(sc[n][i], capped, ca, cb);
                    sc[n][2 + i] = mw_score(sc[n][2 + i], capped, ca, cb);
                    if (!plain) {
                        const int e = e0 + n * 8 + (lane & 3) * 2 + i, p = e < kept ? e : e + gap;
                        const bool first_kept = p < keep_first;
                        if (!(e < n_keys && p <= p_lo && (p >= in_lo || first_kept))) sc[n][i] = -INFINITY;
                        if (!(e < n_keys && p <= p_hi && (p >= in_hi || first_kept))) sc[n][2 + i] = -INFINITY;
                    }
                    c_lo = fmaxf(c_lo, sc[n][i]);
                    c_hi = fmaxf(c_hi, sc[n][2 + i]);
                }
            }
            c_lo = fmaxf(c_lo, __shfl_xor_sync(0xffffffffu, c_lo, 1));
            c_lo = fmaxf(c_lo, __shfl_xor_sync(0xffffffffu, c_lo, 2));
            c_hi = fmaxf(c_hi, __shfl_xor_sync(0xffffffffu, c_hi, 1));
            c_hi = fmaxf(c_hi, __shfl_xor_sync(0xffffffffu, c_hi, 2));
            const float n_lo = fmaxf(m_lo, c_lo), n_hi = fmaxf(m_hi, c_hi);
            // a row that has seen no key yet keeps its zero sums (2^(-inf - -inf) is avoided)
            const float z_lo = n_lo == -INFINITY ? 0.f : n_lo, z_hi = n_hi == -INFINITY ? 0.f : n_hi;
            const float f_lo = mw_exp2(m_lo - z_lo), f_hi = mw_exp2(m_hi - z_hi);
            float s_lo = 0.f, s_hi = 0.f;
#pragma unroll
            for (int n = 0; n < 4; ++n) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    sc[n][i] = mw_exp2(sc[n][i] - z_lo);
                    sc[n][2 + i] = mw_exp2(sc[n][2 + i] - z_hi);
                    s_lo += sc[n][i];
                    s_hi += sc[n][2 + i];
                }
            }
            l_lo = l_lo * f_lo + s_lo;                    // each lane its own part of the row's sum
            l_hi = l_hi * f_hi + s_hi;
            if (__any_sync(0xffffffffu, n_lo != m_lo || n_hi != m_hi)) {
#pragma unroll
                for (int n = 0; n < VT; ++n) { o[n][0] *= f_lo; o[n][1] *= f_lo; o[n][2] *= f_hi; o[n][3] *= f_hi; }
            }
            m_lo = n_lo;
            m_hi = n_hi;
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const uint32_t a0 = mw_pack(sc[2 * j][0], sc[2 * j][1]), a1 = mw_pack(sc[2 * j][2], sc[2 * j][3]);
                const uint32_t a2 = mw_pack(sc[2 * j + 1][0], sc[2 * j + 1][1]), a3 = mw_pack(sc[2 * j + 1][2], sc[2 * j + 1][3]);
                const int vrow = j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
                const uint32_t v_addr = sv_addr + (uint32_t)((vrow * vp + (lane >> 4) * 8) * 2);
#pragma unroll
                for (int n2 = 0; n2 < VT / 2; ++n2) {
                    uint32_t b0_, b1_, b2_, b3_;
                    mw_ldmatrix_x4_trans(v_addr + n2 * 32, b0_, b1_, b2_, b3_);
                    mw_mma(o[n2 * 2], a0, a1, a2, a3, b0_, b1_);
                    mw_mma(o[n2 * 2 + 1], a0, a1, a2, a3, b2_, b3_);
                }
            }
        }
        __syncthreads();                                   // the buffer may be filled again
    }
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
    const float i_lo = 1.0f / l_lo, i_hi = 1.0f / l_hi;
    float* dst = sums + ((size_t)(t0 + r0 - slab0) * n_heads + h) * total + c0;
    const size_t pitch = (size_t)n_heads * total;
#pragma unroll
    for (int n = 0; n < VT; ++n) {
        const int d = n * 8 + (lane & 3) * 2;
        if (d < cw) {
            if (row_lo < rows) *reinterpret_cast<float2*>(dst + row_lo * pitch + d) = make_float2(o[n][0] * i_lo, o[n][1] * i_lo);
            if (row_hi < rows) *reinterpret_cast<float2*>(dst + row_hi * pitch + d) = make_float2(o[n][2] * i_hi, o[n][3] * i_hi);
        }
    }
}

// out[t, h, d] = sum_g mix[h, g] sums[t, g, c(h) * v_dim + d]; a thread per (row, kv head, d), the heads of its group
template <int GROUP>
__global__ void __launch_bounds__(256)
mixed_sum_kernel(const float* __restrict__ sums, const float* __restrict__ mix, __nv_bfloat16* __restrict__ out, int n_rows,
                 int n_heads, int n_kv_heads, int v_dim) {
    chain_release();
    chain_wait();
    extern __shared__ float smix[];                        // [n_heads][n_heads]
    for (int e = threadIdx.x; e < n_heads * n_heads; e += blockDim.x) smix[e] = mix[e];
    __syncthreads();
    const int total = n_kv_heads * v_dim, group = n_heads / n_kv_heads;
    const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long)n_rows * total) return;
    const int t = (int)(i / total), col = (int)(i % total), c = col / v_dim, d = col % v_dim;
    const float* src = sums + (size_t)t * n_heads * total + col;
    for (int g0 = 0; g0 < group; g0 += GROUP) {
        float acc[GROUP];
#pragma unroll
        for (int j = 0; j < GROUP; ++j) acc[j] = 0.f;
        const float* mrow = smix + (size_t)(c * group + g0) * n_heads;
#pragma unroll 8
        for (int g = 0; g < n_heads; ++g) {
            const float x = src[(size_t)g * total];
#pragma unroll
            for (int j = 0; j < GROUP; ++j) acc[j] = fmaf(mrow[j * n_heads + g], x, acc[j]);
        }
#pragma unroll
        for (int j = 0; j < GROUP; ++j) out[((size_t)t * n_heads + c * group + g0 + j) * v_dim + d] = __float2bfloat16_rn(acc[j]);
    }
}

// ---------------------------------------------------------------- single tokens
static size_t mw_step_smem(int n_heads, int n_kv_heads, int dim, int v_dim, int buffers) {
    const int group = n_heads / n_kv_heads, tiles = n_kv_heads * ((group + 15) / 16), m_rows = (n_heads + 15) / 16 * 16;
    return ((size_t)tiles * 16 * (dim + 8) + (size_t)buffers * kMwChunk * (n_kv_heads * (dim + v_dim) + 16) + (size_t)m_rows * (kMwChunk + 8)) * 2 +
           ((size_t)kMwMaxHeads * (kMwChunk + 1) + 3 * kMwMaxHeads) * 4;
}

// NT: value n-tiles of eight columns a warp accumulates at most; MT: tiles of sixteen heads.
template <int NT, int MT>
__global__ void __launch_bounds__(kMwStepWarps * 32)
mixed_step_kernel(const __nv_bfloat16* __restrict__ q, int q_row_stride, const __nv_bfloat16* __restrict__ k_cache,
                  const __nv_bfloat16* __restrict__ v_cache, const float* __restrict__ factor, float softcap,
                  const int* __restrict__ tok_pos, const int* __restrict__ seq_slot, const int* __restrict__ page_table,
                  int max_pages, int page_size, float* __restrict__ partial, int n_heads, int n_kv_heads, int dim, int v_dim,
                  int window, int keep_first, int splits, int buffers) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) unsigned char mw_smem[];
    const int s = blockIdx.y, split = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = tok_pos[s];
    const int first = window > 0 ? max(0, pos + 1 - window) : 0;
    const int kept = min(keep_first, first), gap = first - kept, n_keys = pos + 1 - gap;
    const int n_chunks = (n_keys + kMwChunk - 1) / kMwChunk, per = (n_chunks + splits - 1) / splits;
    const int chunk0 = split * per, chunk1 = min(n_chunks, chunk0 + per);
    const int group = n_heads / n_kv_heads, sub = (group + 15) / 16, tiles = n_kv_heads * sub;
    const int kw = n_kv_heads * dim, total = n_kv_heads * v_dim;
    const int qp = dim + 8, kp = kw + 8, vp = total + 8, pp = kMwChunk + 8;
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(mw_smem);          // [tiles][16][dim + 8]
    __nv_bfloat16* sk = sq + (size_t)tiles * 16 * qp;                        // [buffers][32][kw + 8]
    __nv_bfloat16* sv = sk + (size_t)buffers * kMwChunk * kp;                // [buffers][32][total + 8]
    __nv_bfloat16* sp = sv + (size_t)buffers * kMwChunk * vp;                // [16 MT][32 + 8] the chunk's weights
    float* ss = reinterpret_cast<float*>(sp + (size_t)MT * 16 * pp);         // [heads][33] scores
    float* sm = ss + (size_t)kMwMaxHeads * (kMwChunk + 1);                   // running maxima, normalisers, corrections
    float* sl = sm + kMwMaxHeads;
    float* scorr = sl + kMwMaxHeads;
    const int* pages = page_table + (size_t)seq_slot[s] * max_pages;
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    auto issue = [&](int chunk, int buf) {
        for (int j = warp; j < kMwChunk; j += kMwStepWarps) {
            __nv_bfloat16* dk = sk + ((size_t)buf * kMwChunk + j) * kp;
            __nv_bfloat16* dv = sv + ((size_t)buf * kMwChunk + j) * vp;
            const int e = chunk * kMwChunk + j;
            if (e < n_keys) {
                const int p = e < kept ? e : e + gap;
                const size_t row = (size_t)pages[p / page_size] * page_size + (size_t)(p % page_size);
                for (int d8 = lane; d8 < kw / 8; d8 += 32) mw_copy16(dk + d8 * 8, k_cache + row * kw + d8 * 8);
                for (int d8 = lane; d8 < total / 8; d8 += 32) mw_copy16(dv + d8 * 8, v_cache + row * total + d8 * 8);
            } else {
                for (int d8 = lane; d8 < kw / 8; d8 += 32) *reinterpret_cast<uint4*>(dk + d8 * 8) = zero4;
                for (int d8 = lane; d8 < total / 8; d8 += 32) *reinterpret_cast<uint4*>(dv + d8 * 8) = zero4;
            }
        }
        mw_commit();
    };
    if (chunk0 < chunk1) issue(chunk0, 0);
    // query heads of one kv head are the rows of a tile (or two)
    for (int e = threadIdx.x; e < tiles * 16 * (dim / 8); e += blockDim.x) {
        const int tile = e / (16 * (dim / 8)), r = (e / (dim / 8)) % 16, d8 = e % (dim / 8);
        const int g = (tile % sub) * 16 + r, h = (tile / sub) * group + g;
        uint4 v = zero4;
        if (g < group) v = *reinterpret_cast<const uint4*>(q + (size_t)s * q_row_stride + (size_t)h * dim + d8 * 8);
        *reinterpret_cast<uint4*>(sq + ((size_t)tile * 16 + r) * qp + d8 * 8) = v;
    }
    for (int e = threadIdx.x; e < kMwMaxHeads; e += blockDim.x) { sm[e] = -INFINITY; sl[e] = 0.f; scorr[e] = 1.f; }
    for (int e = threadIdx.x; e < MT * 16 * pp; e += blockDim.x) sp[e] = __float2bfloat16_rn(0.f);
    float o[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f; }
    const bool capped = softcap > 0.f;
    const float ca = softcap * kLog2e;
    // a warp's value columns: pairs of n-tiles (sixteen columns) dealt out evenly
    const int pairs = total / 16, pairs_per = (pairs + kMwStepWarps - 1) / kMwStepWarps;
    const int pair0 = warp * pairs_per, n_pairs = max(0, min(pairs_per, pairs - pair0));
    const int row_lo = lane >> 2;
    for (int chunk = chunk0, buf = 0; chunk < chunk1; ++chunk, buf = buffers == 2 ? buf ^ 1 : 0) {
        if (buffers == 2 && chunk + 1 < chunk1) { issue(chunk + 1, buf ^ 1); mw_wait<1>(); } else { mw_wait<0>(); }
        __syncthreads();
        const uint32_t sk_addr = (uint32_t)__cvta_generic_to_shared(sk + (size_t)buf * kMwChunk * kp);
        const uint32_t sv_addr = (uint32_t)__cvta_generic_to_shared(sv + (size_t)buf * kMwChunk * vp);
        for (int task = warp; task < tiles * 4; task += kMwStepWarps) {      // a tile of heads x eight keys
            const int tile = task >> 2, n = task & 3, c = tile / sub;
            const uint32_t qa = (uint32_t)__cvta_generic_to_shared(sq + (size_t)tile * 16 * qp);
            float sc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
            for (int k0 = 0; k0 < dim; k0 += 16) {
                uint32_t a0, a1, a2, a3, b0, b1;
                mw_ldmatrix_x4(qa + (uint32_t)(((lane & 15) * qp + k0 + (lane >> 4) * 8) * 2), a0, a1, a2, a3);
                mw_ldmatrix_x2(sk_addr + (uint32_t)(((n * 8 + (lane & 7)) * kp + c * dim + k0 + ((lane >> 3) & 1) * 8) * 2), b0, b1);
                mw_mma(sc, a0, a1, a2, a3, b0, b1);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int g = (tile % sub) * 16 + row_lo + (i >> 1) * 8, key = n * 8 + (lane & 3) * 2 + (i & 1);
                if (g < group) {
                    const int h = c * group + g;
                    const float cb = capped ? 2.0f * kLog2e * factor[h] / softcap : kLog2e * factor[h];
                    ss[h * (kMwChunk + 1) + key] = chunk * kMwChunk + key < n_keys ? mw_score(sc[i], capped, ca, cb) : -INFINITY;
                }
            }
        }
        __syncthreads();
        for (int h = warp; h < n_heads; h += kMwStepWarps) {
            const float x = ss[h * (kMwChunk + 1) + lane];                   // a chunk has at least one key
            const float m_old = sm[h], m_new = fmaxf(m_old, warp_max(x));
            const float p = mw_exp2(x - m_new), corr = mw_exp2(m_old - m_new), sum = warp_sum(p);
            sp[h * pp + lane] = __float2bfloat16_rn(p);
            if (lane == 0) { sm[h] = m_new; sl[h] = sl[h] * corr + sum; scorr[h] = corr; }
        }
        __syncthreads();
        const uint32_t sp_addr = (uint32_t)__cvta_generic_to_shared(sp);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float f_lo = m * 16 + row_lo < n_heads ? scorr[m * 16 + row_lo] : 1.f;
            const float f_hi = m * 16 + row_lo + 8 < n_heads ? scorr[m * 16 + row_lo + 8] : 1.f;
#pragma unroll
            for (int n = 0; n < NT; ++n) { o[m][n][0] *= f_lo; o[m][n][1] *= f_lo; o[m][n][2] *= f_hi; o[m][n][3] *= f_hi; }
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            uint32_t a[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
                mw_ldmatrix_x4(sp_addr + (uint32_t)(((m * 16 + (lane & 15)) * pp + j * 16 + (lane >> 4) * 8) * 2), a[m][0], a[m][1], a[m][2], a[m][3]);
#pragma unroll
            for (int n2 = 0; n2 < NT / 2; ++n2) {      // (a pair beyond the warp's computes the last one again, for nothing)
                uint32_t b0, b1, b2, b3;
                const int vrow = j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
                mw_ldmatrix_x4_trans(sv_addr + (uint32_t)((vrow * vp + min(pair0 + n2, pairs - 1) * 16 + (lane >> 4) * 8) * 2), b0, b1, b2, b3);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mw_mma(o[m][n2 * 2], a[m][0], a[m][1], a[m][2], a[m][3], b0, b1);
                    mw_mma(o[m][n2 * 2 + 1], a[m][0], a[m][1], a[m][2], a[m][3], b2, b3);
                }
            }
        }
        if (buffers == 1 && chunk + 1 < chunk1) { __syncthreads(); issue(chunk + 1, 0); }
        else __syncthreads();                                                // buffer, scores and weights may be written again
    }
    // [(sequence, split)][heads][total] sums, then [heads] maxima and [heads] normalisers
    float* dst = partial + ((size_t)s * splits + split) * n_heads * (total + 2);
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            if (n / 2 >= n_pairs) continue;
            const int col = pair0 * 16 + n * 8 + (lane & 3) * 2, h = m * 16 + row_lo;
            if (h < n_heads) *reinterpret_cast<float2*>(dst + (size_t)h * total + col) = make_float2(o[m][n][0], o[m][n][1]);
            if (h + 8 < n_heads) *reinterpret_cast<float2*>(dst + (size_t)(h + 8) * total + col) = make_float2(o[m][n][2], o[m][n][3]);
        }
    __syncthreads();
    for (int h = threadIdx.x; h < n_heads; h += blockDim.x) {
        dst[(size_t)n_heads * total + h] = sm[h];
        dst[(size_t)n_heads * total + n_heads + h] = sl[h];
    }
}

// Block = (sequence, 32 value columns of one kv head or across them): the runs' sums in order, normalised, mixed.
// 256 threads = 32 columns x 8 parts of the heads; the parts are added in order.
constexpr int kMergeCols = 32, kMergeParts = 8, kMwMaxSplits = 64;
template <int GROUP>
__global__ void __launch_bounds__(kMergeCols * kMergeParts)
mixed_merge_kernel(const float* __restrict__ partial, const float* __restrict__ mix, __nv_bfloat16* __restrict__ out, int n_heads,
                   int n_kv_heads, int v_dim, int splits) {
    chain_release();
    chain_wait();
    extern __shared__ float msm[];                         // [splits][heads] factors, then [parts][GROUP][32] sums
    const int s = blockIdx.y, total = n_kv_heads * v_dim, group = n_heads / n_kv_heads;
    const size_t pitch = (size_t)n_heads * (total + 2);
    const float* src = partial + (size_t)s * splits * pitch;
    float* fac = msm;
    float* red = msm + splits * n_heads;
    // a warp per head, lanes over the runs: factors that turn each run's sums into parts of the normalised row
    for (int h = threadIdx.x / 32; h < n_heads; h += kMergeCols * kMergeParts / 32) {
        const int k0 = threadIdx.x & 31, k1 = k0 + 32;
        const float* stat = src + (size_t)n_heads * total + h;
        const float m0 = k0 < splits ? stat[k0 * pitch] : -INFINITY, m1 = k1 < splits ? stat[k1 * pitch] : -INFINITY;
        const float l0 = k0 < splits ? stat[k0 * pitch + n_heads] : 0.f, l1 = k1 < splits ? stat[k1 * pitch + n_heads] : 0.f;
        const float M = warp_max(fmaxf(m0, m1)), e0 = mw_exp2(m0 - M), e1 = mw_exp2(m1 - M);          // 0 for a run without keys
        const float inv = 1.0f / warp_sum(fmaf(l0, e0, l1 * e1));
        if (k0 < splits) fac[k0 * n_heads + h] = e0 * inv;
        if (k1 < splits) fac[k1 * n_heads + h] = e1 * inv;
    }
    __syncthreads();
    const int lane = threadIdx.x % kMergeCols, part = threadIdx.x / kMergeCols;
    const int col = blockIdx.x * kMergeCols + lane;
    const bool live = col < total;
    const int c = live ? col / v_dim : 0, d = live ? col % v_dim : 0;
    for (int g0 = 0; g0 < group; g0 += GROUP) {
        float acc[GROUP];
#pragma unroll
        for (int j = 0; j < GROUP; ++j) acc[j] = 0.f;
        if (live)
#pragma unroll 2
            for (int g = part; g < n_heads; g += kMergeParts) {
                float x = 0.f;
#pragma unroll 16
                for (int k = 0; k < splits; ++k) x = fmaf(src[k * pitch + (size_t)g * total + col], fac[k * n_heads + g], x);
#pragma unroll
                for (int j = 0; j < GROUP; ++j) acc[j] = fmaf(mix[(size_t)(c * group + g0 + j) * n_heads + g], x, acc[j]);
            }
#pragma unroll
        for (int j = 0; j < GROUP; ++j) red[(part * GROUP + j) * kMergeCols + lane] = acc[j];
        __syncthreads();
        for (int j = part; j < GROUP; j += kMergeParts) {
            float y = 0.f;
#pragma unroll
            for (int p = 0; p < kMergeParts; ++p) y += red[(p * GROUP + j) * kMergeCols + lane];
            if (live) out[((size_t)s * n_heads + c * group + g0 + j) * v_dim + d] = __float2bfloat16_rn(y);
        }
        __syncthreads();
    }
}

static int mw_group_part(int group) { return group % 8 == 0 ? 8 : group % 4 == 0 ? 4 : group % 2 == 0 ? 2 : 1; }
static bool mw_sizes_ok(int n_heads, int n_kv_heads, int dim, int v_dim) {
    return n_heads > 0 && n_heads <= kMwMaxHeads && n_kv_heads > 0 && n_heads % n_kv_heads == 0 && dim > 0 && dim % 16 == 0 &&
           dim <= 256 && v_dim > 0 && v_dim % 8 == 0 && (n_kv_heads * v_dim) % 16 == 0;
}
constexpr size_t kMwSmemLimit = 220 * 1024;

}  // namespace mdma

using namespace mdma;

extern "C" {

// out [tokens][heads * v_dim]; sums: slab_tokens * heads * kv_heads * v_dim floats of scratch
int mdma_mixed_weights_rows(const void* q, int q_row_stride, const void* k_cache, const void* v_cache, const float* mix,
                            const float* factor, float softcap, const int* seq_start, const int* seq_pos0, const int* seq_slot,
                            const int* page_table, int max_pages, int page_size, void* out, float* sums, int slab_tokens,
                            int n_tokens, int n_seqs, int max_new, int n_heads, int n_kv_heads, int dim, int v_dim, int window,
                            int keep_first, cudaStream_t stream) {
    MDMA_REQUIRE(mw_sizes_ok(n_heads, n_kv_heads, dim, v_dim), "mixed_weights_rows: %d/%d heads of %d/%d are not a geometry this kernel takes", n_heads, n_kv_heads, dim, v_dim);
    MDMA_REQUIRE(mix && factor && sums && page_table && page_size > 0 && max_pages > 0 && window >= 0 && keep_first >= 0 && slab_tokens > 0,
                 "mixed_weights_rows: bad arguments");
    MDMA_REQUIRE(n_seqs <= 65535 && q_row_stride % 8 == 0, "mixed_weights_rows: too many sequences, or query rows that do not start on 16 bytes");
    MDMA_REQUIRE((((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)sums) & 15) == 0, "mixed_weights_rows: pointers must be 16-byte aligned");
    if (n_tokens == 0 || n_seqs == 0) return 0;
    const int group = n_heads / n_kv_heads, total = n_kv_heads * v_dim;
    const int heads_per_block = group % 4 == 0 ? 4 : group % 2 == 0 ? 2 : 1;
    const int block_rows = kMwWarps / heads_per_block * kMwTile;
    const int parts = (total + 255) / 256;
    const int cols = ((total + parts - 1) / parts + 15) / 16 * 16;
    const int gp = mw_group_part(group);
    for (int slab0 = 0; slab0 < n_tokens; slab0 += slab_tokens) {
        const int slab1 = slab0 + slab_tokens < n_tokens ? slab0 + slab_tokens : n_tokens;
        const int most = max_new < slab1 - slab0 ? max_new : slab1 - slab0;
        dim3 grid((most + block_rows - 1) / block_rows, (n_heads / heads_per_block) * parts, n_seqs);
#define MDMA_MW_ROWS(VT, KD)                                                                                                 \
    do {                                                                                                                     \
        static bool raised = false;                                                                                          \
        if (!raised) { cudaFuncSetAttribute(mixed_rows_kernel<VT, KD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMwSmemLimit); raised = true; } \
        launch_chained(mixed_rows_kernel<VT, KD>, grid, dim3(kMwWarps * 32), mw_rows_smem(dim, VT), stream, (const __nv_bfloat16*)q, \
                       q_row_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, factor, softcap, seq_start, \
                       seq_pos0, seq_slot, page_table, max_pages, page_size, sums, n_heads, n_kv_heads, dim, v_dim, window,  \
                       keep_first, heads_per_block, cols, slab0, slab1);                                                     \
    } while (0)
        if (cols <= 64) MDMA_MW_ROWS(8, 0);
        else if (cols <= 128) MDMA_MW_ROWS(16, 0);
        else if (dim == 128) MDMA_MW_ROWS(32, 8);
        else MDMA_MW_ROWS(32, 0);
#undef MDMA_MW_ROWS
        MDMA_LAUNCH_OK("mixed_weights_rows");
        const long items = (long)(slab1 - slab0) * total;
        const size_t mix_bytes = (size_t)n_heads * n_heads * sizeof(float);
#define MDMA_MW_SUM(G)                                                                                                       \
    launch_chained(mixed_sum_kernel<G>, dim3((unsigned)((items + 255) / 256)), dim3(256), mix_bytes, stream, (const float*)sums, mix, \
                   (__nv_bfloat16*)out + (size_t)slab0 * n_heads * v_dim, slab1 - slab0, n_heads, n_kv_heads, v_dim)
        if (gp == 8) MDMA_MW_SUM(8); else if (gp == 4) MDMA_MW_SUM(4); else if (gp == 2) MDMA_MW_SUM(2); else MDMA_MW_SUM(1);
#undef MDMA_MW_SUM
        MDMA_LAUNCH_OK("mixed_weights_sum");
    }
    return 0;
}

// Whether the single-token kernel takes this geometry (1 or 2: buffers of staged keys), or 0.
int mdma_mixed_weights_step_fits(int n_heads, int n_kv_heads, int dim, int v_dim) {
    if (!mw_sizes_ok(n_heads, n_kv_heads, dim, v_dim)) return 0;
    const int pairs_per = (n_kv_heads * v_dim / 16 + kMwStepWarps - 1) / kMwStepWarps;
    if (pairs_per > 8) return 0;
    if (mw_step_smem(n_heads, n_kv_heads, dim, v_dim, 2) <= kMwSmemLimit) return 2;
    return mw_step_smem(n_heads, n_kv_heads, dim, v_dim, 1) <= kMwSmemLimit ? 1 : 0;
}

// One token per sequence; partial: n_seqs * splits * heads * (kv_heads * v_dim + 2) floats
int mdma_mixed_weights_step(const void* q, int q_row_stride, const void* k_cache, const void* v_cache, const float* mix,
                            const float* factor, float softcap, const int* tok_pos, const int* seq_slot, const int* page_table,
                            int max_pages, int page_size, void* out, float* partial, int splits, int n_seqs, int n_heads,
                            int n_kv_heads, int dim, int v_dim, int window, int keep_first, cudaStream_t stream) {
    const int buffers = mdma_mixed_weights_step_fits(n_heads, n_kv_heads, dim, v_dim);
    MDMA_REQUIRE(buffers > 0, "mixed_weights_step: %d/%d heads of %d/%d are not a geometry this kernel takes", n_heads, n_kv_heads, dim, v_dim);
    MDMA_REQUIRE(mix && factor && partial && page_table && page_size > 0 && max_pages > 0 && window >= 0 && keep_first >= 0 &&
                 splits >= 1 && splits <= kMwMaxSplits, "mixed_weights_step: bad arguments");
    MDMA_REQUIRE(n_seqs <= 65535 && q_row_stride % 8 == 0, "mixed_weights_step: too many sequences, or query rows that do not start on 16 bytes");
    MDMA_REQUIRE((((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)partial) & 15) == 0, "mixed_weights_step: pointers must be 16-byte aligned");
    if (n_seqs == 0) return 0;
    const int total = n_kv_heads * v_dim, group = n_heads / n_kv_heads;
    const int pairs_per = (total / 16 + kMwStepWarps - 1) / kMwStepWarps;
    const size_t smem = mw_step_smem(n_heads, n_kv_heads, dim, v_dim, buffers);
#define MDMA_MW_STEP(NT, MT)                                                                                                 \
    do {                                                                                                                     \
        static bool raised = false;                                                                                          \
        if (!raised) { cudaFuncSetAttribute(mixed_step_kernel<NT, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMwSmemLimit); raised = true; } \
        launch_chained(mixed_step_kernel<NT, MT>, dim3(splits, n_seqs), dim3(kMwStepWarps * 32), smem, stream, (const __nv_bfloat16*)q, \
                       q_row_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, factor, softcap, tok_pos, \
                       seq_slot, page_table, max_pages, page_size, partial, n_heads, n_kv_heads, dim, v_dim, window,         \
                       keep_first, splits, buffers);                                                                         \
    } while (0)
    if (n_heads <= 16) {
        if (pairs_per <= 2) MDMA_MW_STEP(4, 1); else if (pairs_per <= 4) MDMA_MW_STEP(8, 1); else MDMA_MW_STEP(16, 1);
    } else {
        if (pairs_per <= 2) MDMA_MW_STEP(4, 2); else if (pairs_per <= 4) MDMA_MW_STEP(8, 2); else MDMA_MW_STEP(16, 2);
    }
#undef MDMA_MW_STEP
    MDMA_LAUNCH_OK("mixed_weights_step");
    const int gp = mw_group_part(group);
    const size_t merge_smem = ((size_t)splits * n_heads + (size_t)kMergeParts * gp * kMergeCols) * sizeof(float);
#define MDMA_MW_MERGE(G)                                                                                                     \
    launch_chained(mixed_merge_kernel<G>, dim3((total + kMergeCols - 1) / kMergeCols, n_seqs), dim3(kMergeCols * kMergeParts), \
                   merge_smem, stream, (const float*)partial, mix, (__nv_bfloat16*)out, n_heads, n_kv_heads, v_dim, splits)
    if (gp == 8) MDMA_MW_MERGE(8); else if (gp == 4) MDMA_MW_MERGE(4); else if (gp == 2) MDMA_MW_MERGE(2); else MDMA_MW_MERGE(1);
#undef MDMA_MW_MERGE
    MDMA_LAUNCH_OK("mixed_weights_merge");
    return 0;
}

}  // extern "C"
