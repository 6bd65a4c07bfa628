// A matrix memory with exponential gates per head (mLSTM).
//
// Per head, with q, k [dim] (q times a constant) and v [vdim] of a token and its two gate inputs zi, zf:
//     i = cap tanh((zi + bi) / cap),   f = log sigmoid(cap tanh((zf + bf) / cap))       the gates' logarithms
//     m_t = max(f + m_(t-1), i),  m_0 = 0
//     S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T        S [dim][vdim] from zero
//     n_t = e^(f + m_(t-1) - m_t) n_(t-1) + e^(i - m_t) k            n [dim] from zero
//     o_t = S_t^T q / (max(|n_t . q|, e^(-m_t)) + 1e-6)
// all in float.  The projections come as float rows [.. q | k | v | zi | zf ..].
//
// The columns of S do not touch one another: a block owns one (sequence, head, part of the columns).  Every part keeps
// n and m of its own, so that no block reads what another of the same launch writes.  A state row:
//     S [heads][dim][vdim], then [heads][parts][pitch]: n [dim], m, one unused word; pitch a multiple of four.
//
// matrix_memory_scan: row by row in one fixed order (the 32-bit engine, short portions).
//
// matrix_memory_chunk: kMemChunk rows at a time.  With b_r the sum of f over the chunk's rows up to r, a_r = i_r - b_r and
// M_r = max(m, a_0 .. a_r) (m: at the chunk's start), every exponent is a difference to M: m_r = b_r + M_r,
//     o_r = (e^(m - M_r) S^T q_r + sum_(j <= r) e^(a_j - M_r) (q_r . k_j) v_j) / (max(|n_r . q_r|, e^(-m_r)) + 1e-6),
//     n_r . q_r = e^(m - M_r) n . q_r + sum_(j <= r) e^(a_j - M_r) (q_r . k_j),
// and at the chunk's end, with M its last M_r,  S <- e^(m - M) S + sum_j e^(a_j - M) k_j v_j^T, n likewise, m <- b + M.
// Long sequences are cut into runs of `run_rows` rows walked side by side: pass kMemLocal walks every run but the last
// from nothing (m = -infinity) and leaves S, n, m and the run's sum of f in scratch; pass kMemFrom starts run r from the
// sequence's state and the runs before it, each times its share e^(its m + the f of the runs after it - m of the start).
//
// matrix_memory_token: steps of one row a sequence, a block per (sequence, head), from the projection row (or the partial
// sums of a K-split product) to the normed, gated head: o_h / sqrt(mean(o_h^2) + eps) * w * sigmoid(g) * out_scale.
#include "common.cuh"
#include "float4.cuh"

namespace mdma {

constexpr int kMemMaxDim = 256, kMemMaxRuns = 256;
constexpr float kMemFloor = 1e-6f;

struct MemInput {
    const float* proj; int stride;
    int q_col, k_col, v_col, i_col, f_col;
    const void* i_bias; const void* f_bias; int bias_dtype;
    float cap, q_scale;
};
struct MemState {
    float* rows; size_t stride;
    int parts, pitch;              // parts of the columns, floats of a part's n, m and spare word
};
__device__ __forceinline__ float mem_bias(const void* b, int dtype, int h) {
    return dtype == kF32 ? reinterpret_cast<const float*>(b)[h] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(b)[h]);
}
__device__ __forceinline__ float mem_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ void mem_gates(float zi, float zf, float cap, float& li, float& lf) {
    li = cap * tanhf(zi / cap);
    lf = mem_log_sigmoid(cap * tanhf(zf / cap));
}
__device__ __forceinline__ void mem_row_gates(const MemInput& in, int t, int h, float& li, float& lf) {
    const float* row = in.proj + (size_t)t * in.stride;
    mem_gates(row[in.i_col + h] + mem_bias(in.i_bias, in.bias_dtype, h), row[in.f_col + h] + mem_bias(in.f_bias, in.bias_dtype, h), in.cap, li, lf);
}

// ---------------------------------------------------------------- row by row
__global__ void __launch_bounds__(256)
matrix_memory_scan_kernel(const MemInput in, const int* __restrict__ seq_start, const int* __restrict__ seq_slot, const MemState state,
                          float* __restrict__ out, int heads, int dim, int vdim, int cols) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float mem_sm[];
    const int s = blockIdx.x, h = blockIdx.y, part = blockIdx.z;
    const int c0 = part * cols, cw = min(cols, vdim - c0);
    const int t0 = seq_start[s], t1 = seq_start[s + 1];
    if (t1 <= t0) return;
    float* S = mem_sm;                       // [dim][cols]
    float* sn = S + (size_t)dim * cols;      // [dim] each
    float* sq = sn + dim;
    float* sk = sq + dim;
    float* sv = sk + dim;                    // [cols]
    float* red = sv + cols;                  // [256]
    float* size = red + 256;                 // [1]
    float* row_state = state.rows + (size_t)seq_slot[s] * state.stride;
    float* st = row_state + (size_t)h * dim * vdim;
    float* nm = row_state + (size_t)heads * dim * vdim + ((size_t)h * state.parts + part) * state.pitch;
    for (int e = threadIdx.x; e < dim * cw; e += blockDim.x) S[(e / cw) * cols + e % cw] = st[(size_t)(e / cw) * vdim + c0 + e % cw];
    for (int e = threadIdx.x; e < dim; e += blockDim.x) sn[e] = nm[e];
    float m = nm[dim];
    const int groups = blockDim.x / cw;      // cw <= blockDim.x
    const int r = threadIdx.x / cw, j = threadIdx.x % cw;
    for (int t = t0; t < t1; ++t) {
        const float* row = in.proj + (size_t)t * in.stride;
        float li, lf;
        mem_row_gates(in, t, h, li, lf);
        const float m_new = fmaxf(lf + m, li);
        const float keep = expf(lf + m - m_new), take = expf(li - m_new);
        m = m_new;
        for (int e = threadIdx.x; e < dim; e += blockDim.x) {
            const float kv = row[in.k_col + h * dim + e];
            sq[e] = row[in.q_col + h * dim + e] * in.q_scale;
            sk[e] = kv;
            sn[e] = fmaf(keep, sn[e], take * kv);
        }
        for (int e = threadIdx.x; e < cw; e += blockDim.x) sv[e] = row[in.v_col + h * vdim + c0 + e];
        __syncthreads();
        if (r < groups) {
            const float vj = take * sv[j];
            float acc = 0.f;
            for (int i = r; i < dim; i += groups) {
                const float x = fmaf(keep, S[i * cols + j], sk[i] * vj);
                S[i * cols + j] = x;
                acc = fmaf(x, sq[i], acc);
            }
            red[r * cw + j] = acc;
        }
        if (threadIdx.x < 32) {
            float nq = 0.f;
            for (int e = threadIdx.x; e < dim; e += 32) nq = fmaf(sn[e], sq[e], nq);
            nq = warp_sum(nq);
            if (threadIdx.x == 0) *size = fmaxf(fabsf(nq), expf(-m)) + kMemFloor;
        }
        __syncthreads();
        if (threadIdx.x < cw) {
            float o = 0.f;
            for (int g = 0; g < groups; ++g) o += red[g * cw + threadIdx.x];
            out[((size_t)t * heads + h) * vdim + c0 + threadIdx.x] = o / *size;
        }
    }
    __syncthreads();
    for (int e = threadIdx.x; e < dim * cw; e += blockDim.x) st[(size_t)(e / cw) * vdim + c0 + e % cw] = S[(e / cw) * cols + e % cw];
    for (int e = threadIdx.x; e < dim; e += blockDim.x) nm[e] = sn[e];
    if (threadIdx.x == 0) nm[dim] = m;
}

// ---------------------------------------------------------------- a chunk of rows at a time
// Block = (sequence or run, head, part of the columns), 256 threads.  Shared memory, floats, rows of a multiple of four:
// S [dimP][colsP] (dimP a multiple of 8), n [dimP]; q, k [kMemChunk][dimP + 4]; v [kMemChunk][colsP];
// A [kMemChunk][kMemChunk + 4]; six numbers a row.  Rows and columns beyond the data are zero.
//   A[i][j] = e^(a_j - M_i) (q_i . k_j), j <= i: a thread owns two rows and two columns; eight threads a row add up n . q.
//   o: a thread owns two rows of four columns.  S: a thread owns eight by four entries.
constexpr int kMemChunk = 32, kMemAPitch = kMemChunk + 4;
enum MemPass : int { kMemWhole = 0, kMemLocal = 1, kMemFrom = 2 };

template <int PASS>
__global__ void __launch_bounds__(256, 2)
matrix_memory_chunk_kernel(const MemInput in, const int* __restrict__ seq_start, const int* __restrict__ seq_slot, const MemState state,
                           float* __restrict__ out, int heads, int dim, int vdim, int cols, int run_rows, int max_runs,
                           float* __restrict__ run_state, size_t unit) {
    chain_release();
    chain_wait();
    extern __shared__ __align__(16) float mem_sm[];
    const int s = PASS == kMemWhole ? blockIdx.x : blockIdx.x / max_runs;
    const int run = PASS == kMemWhole ? 0 : blockIdx.x % max_runs;
    const int h = blockIdx.y, part = blockIdx.z;
    const int c0 = part * cols, cw = min(cols, vdim - c0);
    int t0 = seq_start[s], t1 = seq_start[s + 1];
    const int runs = PASS == kMemWhole ? 1 : (t1 - t0 + run_rows - 1) / run_rows;
    const size_t head_at = (size_t)h * dim * vdim;
    const size_t nm_at = (size_t)heads * dim * vdim + ((size_t)h * state.parts + part) * state.pitch;
    float* row_state = state.rows + (size_t)seq_slot[s] * state.stride;
    float* rs = PASS == kMemWhole ? nullptr : run_state + (size_t)blockIdx.x * unit;
    bool last_run = true;
    if (PASS != kMemWhole) {
        last_run = run == runs - 1;
        if (run >= runs) return;                                          // the whole block leaves together
        if (PASS == kMemLocal && last_run) {                              // the second pass reads the state from here
            for (int e = threadIdx.x; e < dim * cw; e += blockDim.x) {
                const size_t at = head_at + (size_t)(e / cw) * vdim + c0 + e % cw;
                rs[at] = row_state[at];
            }
            for (int e = threadIdx.x; e <= dim; e += blockDim.x) rs[nm_at + e] = row_state[nm_at + e];
            return;
        }
        t0 += run * run_rows;
        t1 = min(t1, t0 + run_rows);
    }
    if (t1 <= t0) return;
    const int dimP = (dim + 7) & ~7, colsP = (cols + 3) & ~3, kd = dimP + 4, cg = colsP >> 2;
    float* S = mem_sm;                                   // [dimP][colsP]
    float* sn = S + (size_t)dimP * colsP;                // [dimP]
    float* sq = sn + dimP;                               // [kMemChunk][kd]
    float* sk = sq + (size_t)kMemChunk * kd;             // [kMemChunk][kd]
    float* sv = sk + (size_t)kMemChunk * kd;             // [kMemChunk][colsP]
    float* sa = sv + (size_t)kMemChunk * colsP;          // [kMemChunk][kMemAPitch]
    float* ra = sa + (size_t)kMemChunk * kMemAPitch;     // a_r
    float* rM = ra + kMemChunk;                          // M_r
    float* rin = rM + kMemChunk;                         // e^(m - M_r)
    float* rfl = rin + kMemChunk;                        // e^(-m_r)
    float* rw = rfl + kMemChunk;                         // e^(a_r - M)
    float* rinv = rw + kMemChunk;                        // one over the size a row is divided by
    float* coef = rinv + kMemChunk;                      // kMemFrom: the shares of the state and of the runs before, [kMemMaxRuns + 4]
    float m, f_sum = 0.f;                                // the same in every thread
    if (PASS == kMemFrom) {
        const float* first = run_state + (size_t)s * max_runs * unit;
        const float* s0 = first + (size_t)(runs - 1) * unit;
        if (threadIdx.x == 0) {
            float top = s0[nm_at + dim], after = 0.f;
            for (int p = 0; p < run; ++p) top = fmaxf(first[(size_t)p * unit + nm_at + dim + 1] + top, first[(size_t)p * unit + nm_at + dim]);
            for (int p = run - 1; p >= 0; --p) {
                coef[1 + p] = expf(first[(size_t)p * unit + nm_at + dim] + after - top);
                after += first[(size_t)p * unit + nm_at + dim + 1];
            }
            coef[0] = expf(s0[nm_at + dim] + after - top);
            coef[kMemMaxRuns + 1] = top;
        }
        __syncthreads();
        m = coef[kMemMaxRuns + 1];
        const bool quads = ((vdim | cw | c0) & 3) == 0 && (head_at & 3) == 0 && (unit & 3) == 0 && ((uintptr_t)run_state & 15) == 0;
        for (int e = threadIdx.x; e < dimP * cg; e += blockDim.x) {
            const int d = e / cg, c = (e % cg) << 2;
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            if (d < dim && c < cw) {
                const size_t at = head_at + (size_t)d * vdim + c0 + c;
                if (quads) {
                    fma4(acc, coef[0], ld4(s0 + at));
#pragma unroll 4
                    for (int p = 0; p < run; ++p) fma4(acc, coef[1 + p], ld4(first + (size_t)p * unit + at));
                } else {
                    float v[4] = {0.f, 0.f, 0.f, 0.f};
                    for (int i = 0; i < 4 && c + i < cw; ++i) {
                        v[i] = coef[0] * s0[at + i];
                        for (int p = 0; p < run; ++p) v[i] = fmaf(coef[1 + p], first[(size_t)p * unit + at + i], v[i]);
                    }
                    acc = make_float4(v[0], v[1], v[2], v[3]);
                }
            }
            st4(S + (size_t)d * colsP + c, acc);
        }
        for (int e = threadIdx.x; e < dimP; e += blockDim.x) {
            float acc = 0.f;
            if (e < dim) {
                acc = coef[0] * s0[nm_at + e];
                for (int p = 0; p < run; ++p) acc = fmaf(coef[1 + p], first[(size_t)p * unit + nm_at + e], acc);
            }
            sn[e] = acc;
        }
    } else {
        const bool from_state = PASS == kMemWhole;
        for (int e = threadIdx.x; e < dimP * colsP; e += blockDim.x) {
            const int d = e / colsP, c = e % colsP;
            S[e] = (from_state && d < dim && c < cw) ? row_state[head_at + (size_t)d * vdim + c0 + c] : 0.f;
        }
        for (int e = threadIdx.x; e < dimP; e += blockDim.x) sn[e] = (from_state && e < dim) ? row_state[nm_at + e] : 0.f;
        m = from_state ? row_state[nm_at + dim] : -INFINITY;
    }
    // every head's part of a row starts on 16 bytes: rows are read four numbers at a time
    const bool vec = (((uintptr_t)in.proj & 15) | (in.stride & 3) | (dim & 3) | (vdim & 3) | (cols & 3) | (in.q_col & 3) | (in.k_col & 3) | (in.v_col & 3)) == 0;
    for (int r0 = t0; r0 < t1; r0 += kMemChunk) {
        const int n = min(kMemChunk, t1 - r0);
        __syncthreads();                                 // the chunk before is done with q, k, v and the rows' numbers
        if (vec) {
            const int d4 = dimP >> 2;
            for (int e = threadIdx.x; e < kMemChunk * d4; e += blockDim.x) {
                const int i = e / d4, d = (e % d4) << 2;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
                if (i < n && d < dim) {
                    const float* row = in.proj + (size_t)(r0 + i) * in.stride + h * dim + d;
                    y = ld4(row + in.k_col);
                    if (PASS != kMemLocal) { x = ld4(row + in.q_col); scale4(x, in.q_scale); }
                }
                st4(sk + i * kd + d, y);
                if (PASS != kMemLocal) st4(sq + i * kd + d, x);
            }
            for (int e = threadIdx.x; e < kMemChunk * cg; e += blockDim.x) {
                const int i = e / cg, c = (e % cg) << 2;
                float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
                if (i < n && c < cw) x = ld4(in.proj + (size_t)(r0 + i) * in.stride + in.v_col + h * vdim + c0 + c);
                st4(sv + i * colsP + c, x);
            }
        } else {
            for (int e = threadIdx.x; e < kMemChunk * dimP; e += blockDim.x) {
                const int i = e / dimP, d = e % dimP;
                const bool have = i < n && d < dim;
                const float* row = in.proj + (size_t)(r0 + i) * in.stride + h * dim + d;
                sk[i * kd + d] = have ? row[in.k_col] : 0.f;
                if (PASS != kMemLocal) sq[i * kd + d] = have ? row[in.q_col] * in.q_scale : 0.f;
            }
            for (int e = threadIdx.x; e < kMemChunk * colsP; e += blockDim.x) {
                const int i = e / colsP, c = e % colsP;
                sv[e] = (i < n && c < cw) ? in.proj[(size_t)(r0 + i) * in.stride + in.v_col + h * vdim + c0 + c] : 0.f;
            }
        }
        // the rows' gates: every warp works them out for itself, a lane a row; the first leaves them in shared memory
        float S_keep, b_last;
        {
            const int lane = threadIdx.x & 31;
            float li = -INFINITY, lf = 0.f;
            if (lane < n) mem_row_gates(in, r0 + lane, h, li, lf);
            float b = lf;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, b, o);
                if (lane >= o) b += x;
            }
            const float a = lane < n ? li - b : -INFINITY;
            float M = fmaxf(a, m);
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, M, o);
                if (lane >= o) M = fmaxf(M, x);
            }
            const float M_last = __shfl_sync(0xffffffffu, M, 31);          // rows beyond the chunk's last change nothing
            b_last = __shfl_sync(0xffffffffu, b, 31);
            S_keep = expf(m - M_last);
            if (threadIdx.x < kMemChunk) {
                ra[lane] = a; rM[lane] = M; rin[lane] = expf(m - M); rfl[lane] = expf(-(b + M)); rw[lane] = expf(a - M_last);
            }
            m = b_last + M_last;
            f_sum += b_last;
        }
        __syncthreads();
        if (PASS != kMemLocal) {
            {   // A: rows 2 ti, 2 ti + 1; columns tj, tj + 16
                const int ti = threadIdx.x >> 4, tj = threadIdx.x & 15;
                const int i0 = 2 * ti, i1 = i0 + 1, j0 = tj, j1 = tj + 16;
                float a00 = 0.f, a01 = 0.f, a10 = 0.f, a11 = 0.f;
                const float* q0 = sq + i0 * kd; const float* q1 = sq + i1 * kd;
                const float* k0 = sk + j0 * kd; const float* k1 = sk + j1 * kd;
                if (j1 <= i1) {
#pragma unroll 2
                    for (int d = 0; d < dimP; d += 4) {
                        const float4 x0 = ld4(q0 + d), x1 = ld4(q1 + d), y0 = ld4(k0 + d), y1 = ld4(k1 + d);
                        a00 = dot4(x0, y0, a00); a10 = dot4(x1, y0, a10);
                        a01 = dot4(x0, y1, a01); a11 = dot4(x1, y1, a11);
                    }
                } else if (j0 <= i1) {
#pragma unroll 2
                    for (int d = 0; d < dimP; d += 4) {
                        const float4 x0 = ld4(q0 + d), x1 = ld4(q1 + d), y0 = ld4(k0 + d);
                        a00 = dot4(x0, y0, a00); a10 = dot4(x1, y0, a10);
                    }
                }
                const float M0 = rM[i0], M1 = rM[i1], e0 = ra[j0], e1 = ra[j1];
                sa[i0 * kMemAPitch + j0] = j0 <= i0 ? a00 * expf(e0 - M0) : 0.f;
                sa[i1 * kMemAPitch + j0] = j0 <= i1 ? a10 * expf(e0 - M1) : 0.f;
                sa[i0 * kMemAPitch + j1] = j1 <= i0 ? a01 * expf(e1 - M0) : 0.f;
                sa[i1 * kMemAPitch + j1] = j1 <= i1 ? a11 * expf(e1 - M1) : 0.f;
            }
            __syncthreads();
            {   // n . q and the size a row is divided by
                const int i = threadIdx.x >> 3, u = threadIdx.x & 7;
                float nq = 0.f, own = 0.f;
                for (int d = u; d < dimP; d += 8) nq = fmaf(sn[d], sq[i * kd + d], nq);
#pragma unroll
                for (int j = 0; j < kMemChunk / 8; ++j) own += sa[i * kMemAPitch + u + 8 * j];
                nq = fmaf(nq, rin[i], own);
#pragma unroll
                for (int o = 4; o > 0; o >>= 1) nq += __shfl_xor_sync(0xffffffffu, nq, o);
                if (u == 0) rinv[i] = 1.0f / (fmaxf(fabsf(nq), rfl[i]) + kMemFloor);
            }
            __syncthreads();
            for (int tile = threadIdx.x; tile < (kMemChunk / 2) * cg; tile += blockDim.x) {
                const int c = (tile % cg) << 2, i0 = (tile / cg) << 1, i1 = i0 + 1;
                if (i0 >= n) continue;
                const float* q0 = sq + i0 * kd; const float* q1 = sq + i1 * kd;
                float4 o0 = make_float4(0.f, 0.f, 0.f, 0.f), o1 = o0;
#pragma unroll 2
                for (int d = 0; d < dimP; d += 4) {
                    const float4 x0 = ld4(q0 + d), x1 = ld4(q1 + d);
                    const float4 s0 = ld4(S + (size_t)d * colsP + c), s1 = ld4(S + (size_t)(d + 1) * colsP + c);
                    const float4 s2 = ld4(S + (size_t)(d + 2) * colsP + c), s3 = ld4(S + (size_t)(d + 3) * colsP + c);
                    fma4(o0, x0.x, s0); fma4(o0, x0.y, s1); fma4(o0, x0.z, s2); fma4(o0, x0.w, s3);
                    fma4(o1, x1.x, s0); fma4(o1, x1.y, s1); fma4(o1, x1.z, s2); fma4(o1, x1.w, s3);
                }
                scale4(o0, rin[i0]);
                scale4(o1, rin[i1]);
                for (int j = 0; j <= i1; j += 4) {       // A is zero beyond the diagonal, v beyond the chunk's rows
                    const float4 a0 = ld4(sa + i0 * kMemAPitch + j), a1 = ld4(sa + i1 * kMemAPitch + j);
                    const float4 v0 = ld4(sv + j * colsP + c), v1 = ld4(sv + (j + 1) * colsP + c);
                    const float4 v2 = ld4(sv + (j + 2) * colsP + c), v3 = ld4(sv + (j + 3) * colsP + c);
                    fma4(o0, a0.x, v0); fma4(o0, a0.y, v1); fma4(o0, a0.z, v2); fma4(o0, a0.w, v3);
                    fma4(o1, a1.x, v0); fma4(o1, a1.y, v1); fma4(o1, a1.z, v2); fma4(o1, a1.w, v3);
                }
                scale4(o0, rinv[i0]);
                scale4(o1, rinv[i1]);
                float* w0 = out + ((size_t)(r0 + i0) * heads + h) * vdim + c0 + c;
                const float v0[4] = {o0.x, o0.y, o0.z, o0.w}, v1[4] = {o1.x, o1.y, o1.z, o1.w};
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (c + e < cw) {
                        w0[e] = v0[e];
                        if (i1 < n) w0[(size_t)heads * vdim + e] = v1[e];
                    }
            }
            if (PASS == kMemFrom && !last_run && r0 + kMemChunk >= t1) break;      // nobody reads this run's last S
            __syncthreads();                             // every o has read S and n before they change
        }
        for (int tile = threadIdx.x; tile < (dimP >> 3) * cg; tile += blockDim.x) {
            const int c = (tile % cg) << 2, d = (tile / cg) << 3;
            float* Sd = S + (size_t)d * colsP + c;
            float4 acc[8];
#pragma unroll
            for (int r = 0; r < 8; ++r) { acc[r] = ld4(Sd + r * colsP); scale4(acc[r], S_keep); }
#pragma unroll 2
            for (int j = 0; j < n; ++j) {
                float4 vv = ld4(sv + j * colsP + c);
                scale4(vv, rw[j]);
                const float4 ka = ld4(sk + j * kd + d), kb = ld4(sk + j * kd + d + 4);
                fma4(acc[0], ka.x, vv); fma4(acc[1], ka.y, vv); fma4(acc[2], ka.z, vv); fma4(acc[3], ka.w, vv);
                fma4(acc[4], kb.x, vv); fma4(acc[5], kb.y, vv); fma4(acc[6], kb.z, vv); fma4(acc[7], kb.w, vv);
            }
#pragma unroll
            for (int r = 0; r < 8; ++r) st4(Sd + r * colsP, acc[r]);
        }
        for (int d = threadIdx.x; d < dimP; d += blockDim.x) {
            float acc = sn[d] * S_keep;
            for (int j = 0; j < n; ++j) acc = fmaf(rw[j], sk[j * kd + d], acc);
            sn[d] = acc;
        }
    }
    __syncthreads();
    float* to = PASS == kMemLocal ? rs : (last_run ? row_state : nullptr);
    if (to != nullptr) {
        for (int e = threadIdx.x; e < dim * cw; e += blockDim.x) to[head_at + (size_t)(e / cw) * vdim + c0 + e % cw] = S[(e / cw) * colsP + e % cw];
        for (int e = threadIdx.x; e < dim; e += blockDim.x) to[nm_at + e] = sn[e];
        if (threadIdx.x == 0) { to[nm_at + dim] = m; to[nm_at + dim + 1] = f_sum; }
    }
}

// ---------------------------------------------------------------- single tokens
// Block = (sequence, head), 512 threads: a thread owns four neighbouring columns of every `groups`-th row of S.
constexpr int kMemTokThreads = 512, kMemTokRows = 8;

template <typename TW>
__global__ void __launch_bounds__(kMemTokThreads)
matrix_memory_token_kernel(const MemInput in, const float* __restrict__ partial, int splits, size_t split_stride, int row_width, int g_col,
                           const TW* __restrict__ norm_w, const int* __restrict__ seq_slot, const MemState state,
                           __nv_bfloat16* __restrict__ out, int heads, int dim, int vdim, float eps, float out_scale) {
    chain_release();
    chain_wait();
    __shared__ __align__(16) float sq[kMemMaxDim], sk[kMemMaxDim], sv[kMemMaxDim], sg[kMemMaxDim], sn[kMemMaxDim];
    __shared__ __align__(16) float red[kMemTokThreads * 4];
    __shared__ float small[40];
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int quads = vdim >> 2, groups = kMemTokThreads / quads;
    const int c = (tid % quads) << 2, g = tid / quads;
    const bool active = g < groups;
    float* row_state = state.rows + (size_t)seq_slot[s] * state.stride;
    float* st = row_state + (size_t)h * dim * vdim + c;
    float* nm = row_state + (size_t)heads * dim * vdim + (size_t)h * state.parts * state.pitch;
    float4 S[kMemTokRows];
    auto fetch = [&](int d0) {
#pragma unroll
        for (int i = 0; i < kMemTokRows; ++i) {
            const int d = d0 + g + groups * i;
            S[i] = (active && d < dim) ? ld4(st + (size_t)d * vdim) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    fetch(0);                                            // on its way while the row's inputs are put together
    const float* row = in.proj + (size_t)s * in.stride;
    const float* prow = partial + (size_t)s * row_width;
    auto input = [&](int col) -> float {
        if (splits == 0) return row[col];
        float x = 0.f;
#pragma unroll 4
        for (int p = 0; p < splits; ++p) x += prow[(size_t)p * split_stride + col];
        return x;
    };
    const float m_old = nm[dim];
    for (int e = tid; e < 2 * dim + 2 * vdim; e += kMemTokThreads) {
        if (e < dim) sq[e] = input(in.q_col + h * dim + e) * in.q_scale;
        else if (e < 2 * dim) { sk[e - dim] = input(in.k_col + h * dim + e - dim); sn[e - dim] = nm[e - dim]; }
        else if (e < 2 * dim + vdim) sv[e - 2 * dim] = input(in.v_col + h * vdim + e - 2 * dim);
        else sg[e - 2 * dim - vdim] = 1.0f / (1.0f + expf(-input(g_col + h * vdim + e - 2 * dim - vdim)));
    }
    if (tid == kMemTokThreads - 1) {
        float li, lf;
        mem_gates(input(in.i_col + h) + mem_bias(in.i_bias, in.bias_dtype, h), input(in.f_col + h) + mem_bias(in.f_bias, in.bias_dtype, h), in.cap, li, lf);
        const float m_new = fmaxf(lf + m_old, li);
        small[0] = expf(lf + m_old - m_new);
        small[1] = expf(li - m_new);
        small[2] = m_new;
    }
    __syncthreads();
    const float keep = small[0], take = small[1], m = small[2];
    float nq = 0.f;
    for (int d = tid; d < dim; d += kMemTokThreads) {
        const float x = fmaf(keep, sn[d], take * sk[d]);
        for (int p = 0; p < state.parts; ++p) nm[(size_t)p * state.pitch + d] = x;
        nq = fmaf(x, sq[d], nq);
    }
    if (tid < state.parts) nm[(size_t)tid * state.pitch + dim] = m;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 v4 = active ? ld4(sv + c) : acc;
    scale4(v4, take);
    const int step = groups * kMemTokRows;
    for (int d0 = 0; d0 < dim; d0 += step) {
#pragma unroll
        for (int i = 0; i < kMemTokRows; ++i) {
            const int d = d0 + g + groups * i;
            if (active && d < dim) {
                float4 x = S[i];
                scale4(x, keep);
                fma4(x, sk[d], v4);
                st4(st + (size_t)d * vdim, x);
                fma4(acc, sq[d], x);
            }
        }
        if (d0 + step < dim) fetch(d0 + step);
    }
    if (active) st4(red + (size_t)g * vdim + c, acc);
    nq = warp_sum(nq);
    if ((tid & 31) == 0) small[8 + (tid >> 5)] = nq;
    __syncthreads();
    nq = 0.f;
#pragma unroll
    for (int w = 0; w < kMemTokThreads / 32; ++w) nq += small[8 + w];
    const float size = fmaxf(fabsf(nq), expf(-m)) + kMemFloor;
    float o = 0.f;
    if (tid < vdim) {
        for (int i = 0; i < groups; ++i) o += red[(size_t)i * vdim + tid];
        o /= size;
    }
    const float sq_sum = warp_sum(o * o);
    if ((tid & 31) == 0) small[24 + (tid >> 5)] = sq_sum;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < kMemTokThreads / 32; ++w) total += small[24 + w];
    if (tid < vdim)
        out[((size_t)s * heads + h) * vdim + tid] =
            __float2bfloat16_rn(o * (out_scale / sqrtf(total / (float)vdim + eps)) * to_float(norm_w[(size_t)h * vdim + tid]) * sg[tid]);
}

static int mem_cols(int dim, int vdim) {
    int cols = vdim < 64 ? vdim : 64;
    while (cols > 1 && (size_t)dim * cols > 12288) cols = (cols + 1) / 2;
    return cols;
}
static int mem_parts(int dim, int vdim) { const int c = mem_cols(dim, vdim); return (vdim + c - 1) / c; }
static int mem_pitch(int dim) { return (dim + 2 + 3) & ~3; }
static size_t mem_unit(int heads, int dim, int vdim) {
    return (((size_t)heads * ((size_t)dim * vdim + (size_t)mem_parts(dim, vdim) * mem_pitch(dim))) + 3) & ~(size_t)3;
}
static size_t mem_chunk_smem(int dim, int cols) {
    const size_t dimP = (dim + 7) & ~7, colsP = (cols + 3) & ~3;
    return sizeof(float) * (dimP * colsP + dimP + 2 * (size_t)kMemChunk * (dimP + 4) + (size_t)kMemChunk * colsP +
                            (size_t)kMemChunk * kMemAPitch + 6 * kMemChunk + kMemMaxRuns + 4);
}
constexpr size_t kMemSmemMost = 200 * 1024;

}  // namespace mdma

using namespace mdma;

extern "C" {

// Floats of a sequence's state (see above).
long mdma_matrix_memory_floats(int heads, int dim, int vdim) { return (long)mem_unit(heads, dim, vdim); }

// chunked 0: row by row; 1: a chunk of rows at a time, with run_rows > 0 in runs of that many rows side by side
// (`max_runs`: the most runs of a sequence, kMemMaxRuns at most; scratch: n_seqs * max_runs states).  out [rows][heads * vdim].
int mdma_matrix_memory(const float* proj, int stride, int q_col, int k_col, int v_col, int i_col, int f_col, const void* i_bias,
                       const void* f_bias, int bias_dtype, float cap, float q_scale, const int* seq_start, const int* seq_slot,
                       float* state, long state_stride, float* out, int n_seqs, int heads, int dim, int vdim, int chunked,
                       int run_rows, int max_runs, float* scratch, long scratch_floats, cudaStream_t stream) {
    MDMA_REQUIRE(n_seqs >= 0 && heads > 0 && dim > 0 && vdim > 0 && dim <= kMemMaxDim && vdim <= kMemMaxDim,
                 "matrix_memory: heads of %d x %d are beyond the limit %d", dim, vdim, kMemMaxDim);
    MDMA_REQUIRE(heads <= 65535 && cap > 0.f, "matrix_memory: bad sizes");
    if (n_seqs == 0) return 0;
    const MemInput in = {proj, stride, q_col, k_col, v_col, i_col, f_col, i_bias, f_bias, bias_dtype, cap, q_scale};
    const MemState st = {state, (size_t)state_stride, mem_parts(dim, vdim), mem_pitch(dim)};
    const int cols = mem_cols(dim, vdim);
    dim3 grid(n_seqs, heads, st.parts);
    if (!chunked) {
        const size_t smem = sizeof(float) * ((size_t)dim * cols + 3 * (size_t)dim + cols + 256 + 4);
        MDMA_REQUIRE(smem <= kMemSmemMost, "matrix_memory: heads of %d x %d do not fit a block's shared memory", dim, vdim);
        cudaFuncSetAttribute(matrix_memory_scan_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMemSmemMost);
        launch_chained(matrix_memory_scan_kernel, grid, dim3(256), smem, stream, in, seq_start, seq_slot, st, out, heads, dim, vdim, cols);
        MDMA_LAUNCH_OK("matrix_memory (row by row)");
        return 0;
    }
    const size_t smem = mem_chunk_smem(dim, cols), unit = mem_unit(heads, dim, vdim);
    MDMA_REQUIRE(smem <= kMemSmemMost, "matrix_memory: heads of %d x %d do not fit a block's shared memory", dim, vdim);
    if (run_rows > 0) {
        const long slots = (long)n_seqs * max_runs;
        MDMA_REQUIRE(max_runs >= 1 && max_runs <= kMemMaxRuns && scratch != nullptr && scratch_floats >= slots * (long)unit,
                     "matrix_memory: %ld runs (at most %d a sequence) need %ld floats of scratch, %ld given", slots, kMemMaxRuns, slots * (long)unit, scratch_floats);
        grid.x = (unsigned)slots;
    } else {
        max_runs = 1;
    }
#define MDMA_MEM_CHUNK(PASS_, what)                                                                                           \
    cudaFuncSetAttribute(matrix_memory_chunk_kernel<PASS_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMemSmemMost);  \
    launch_chained(matrix_memory_chunk_kernel<PASS_>, grid, dim3(256), smem, stream, in, seq_start, seq_slot, st, out, heads, \
                   dim, vdim, cols, run_rows, max_runs, scratch, unit);                                                       \
    MDMA_LAUNCH_OK(what)
    if (run_rows > 0) {
        MDMA_MEM_CHUNK(kMemLocal, "matrix_memory (runs from nothing)");
        MDMA_MEM_CHUNK(kMemFrom, "matrix_memory (runs from their starts)");
        return 0;
    }
    MDMA_MEM_CHUNK(kMemWhole, "matrix_memory (chunks)");
#undef MDMA_MEM_CHUNK
    return 0;
}

// Whether the single-token kernel takes these sizes.
int mdma_matrix_memory_token_fits(int dim, int vdim) { return dim > 0 && dim <= kMemMaxDim && vdim > 0 && vdim <= kMemMaxDim && vdim % 4 == 0; }

// One token per sequence: the projection rows, or with splits > 0 the sums of `splits` partial rows of row_width floats;
// out [sequences][heads * vdim] bfloat16.
int mdma_matrix_memory_token(const float* proj, int stride, const float* partial, int splits, long split_stride, int row_width, int q_col,
                             int k_col, int v_col, int g_col, int i_col, int f_col, const void* i_bias, const void* f_bias, int bias_dtype,
                             float cap, float q_scale, const void* norm_w, int w_dtype, const int* seq_slot, float* state, long state_stride,
                             void* out, int n_seqs, int heads, int dim, int vdim, float eps, float out_scale, cudaStream_t stream) {
    MDMA_REQUIRE(mdma_matrix_memory_token_fits(dim, vdim), "matrix_memory_token: heads of %d x %d are outside its limits", dim, vdim);
    MDMA_REQUIRE(((uintptr_t)state & 15) == 0 && state_stride % 4 == 0, "matrix_memory_token: state rows must be 16-byte aligned");
    MDMA_REQUIRE(n_seqs >= 0 && heads > 0 && heads <= 65535 && cap > 0.f && (splits == 0 || partial), "matrix_memory_token: bad sizes");
    if (n_seqs == 0) return 0;
    const MemInput in = {proj, stride, q_col, k_col, v_col, i_col, f_col, i_bias, f_bias, bias_dtype, cap, q_scale};
    const MemState st = {state, (size_t)state_stride, mem_parts(dim, vdim), mem_pitch(dim)};
    MDMA_DISPATCH_DTYPE(w_dtype, TW,
        launch_chained(matrix_memory_token_kernel<TW>, dim3(n_seqs, heads), dim3(kMemTokThreads), 0, stream, in, partial, splits,
                       (size_t)split_stride, row_width, g_col, (const TW*)norm_w, seq_slot, st, (__nv_bfloat16*)out, heads, dim, vdim, eps, out_scale));
    MDMA_LAUNCH_OK("matrix_memory_token");
    return 0;
}

}  // extern "C"
