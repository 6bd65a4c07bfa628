// The gated delta rule with a decay per key channel, and the gated norm per head that follows it.
//
// Per head, with unit vectors q (times dim^-1/2) and k [dim], v [vdim], a step size b and decays g [dim] of a token:
//     S <- diag(g) S;   u = b (v - S^T k);   S <- S + k u^T;   o = S^T q          S [dim][vdim] floats per sequence
//
// delta_prepare: from the projections to what enters the recurrence, all in float, a warp per (token, unit): q and k
// heads pass a short causal convolution per channel and silu and become unit vectors, v heads pass convolution and
// silu, decay heads become log g = -exp(A_log) softplus(a + dt_bias), and b = sigmoid(its logit).
//
// delta_token: single tokens of the serving engine, all of the above for one (sequence, head) in one block: the low-rank
// products for the decays and the output gate, convolutions, unit vectors, the recurrence on a state held in registers
// between one read and one write, the gated norm.  It adds up the partial sums a K-split projection left.
//
// delta_scan: row by row, block = (sequence, head, 32 columns of S).  Every thread keeps its part of S in registers for
// all rows of the step; every sum has one fixed order, so the result does not depend on how rows were cut into steps.
// The 32-bit engine's walk, and short portions.
//
// gated_head_rmsnorm: out = o_h / sqrt(mean(o_h^2) + eps) [* w] * act(gate) * scale, per head, act = sigmoid or silu; w is one
// head's (all heads share it) or the whole row's.
#include "delta_rule.cuh"

namespace mdma {

// proj rows [q (kv_heads * dim) | k (kv_heads * dim) | v (heads * vdim) | b (heads)], floats; raw [rows][heads * dim]
// the decays' inputs; q, k [rows][kv_heads * dim], v [rows][heads * vdim], lg [rows][heads * dim], beta [rows][heads]
constexpr int kDeltaPrepWarps = 8;
__global__ void __launch_bounds__(kDeltaPrepWarps * 32)
delta_prepare_kernel(const float* __restrict__ proj, int proj_stride, const float* __restrict__ raw, const void* __restrict__ conv_w,
                     int conv_dtype, int taps, const void* __restrict__ a_log, const void* __restrict__ dt_bias, int vec_dtype,
                     const int* __restrict__ tok_seq, const int* __restrict__ seq_start, const int* __restrict__ seq_slot,
                     const float* __restrict__ state, size_t state_stride, float* __restrict__ q, float* __restrict__ k,
                     float* __restrict__ v, float* __restrict__ lg, float* __restrict__ beta, int heads, int kv_heads,
                     int dim, int vdim, float unit_eps, float q_scale) {
    chain_release();
    chain_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31;
    const int unit = blockIdx.y * kDeltaPrepWarps + (threadIdx.x >> 5);
    if (unit >= 2 * kv_heads + 2 * heads) return;
    const int s = tok_seq[t], t0 = seq_start[s];
    const int qk = kv_heads * dim, channels = 2 * qk + heads * vdim;
    const float* kept = state + (size_t)seq_slot[s] * state_stride;
    if (unit < 2 * kv_heads) {
        const bool is_q = unit < kv_heads;
        const int h = is_q ? unit : unit - kv_heads, c0 = (is_q ? 0 : qk) + h * dim;
        float x[kDeltaMaxDim / 32];
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < kDeltaMaxDim / 32; ++i) {
            const int d = lane + 32 * i;
            x[i] = d < dim ? delta_conv(proj, proj_stride, kept, conv_w, conv_dtype, taps, channels, t, t0, c0 + d) : 0.f;
            sq = fmaf(x[i], x[i], sq);
        }
        const float inv = (is_q ? q_scale : 1.0f) / sqrtf(warp_sum(sq) + unit_eps);
        float* dst = (is_q ? q : k) + (size_t)t * qk + h * dim;
#pragma unroll
        for (int i = 0; i < kDeltaMaxDim / 32; ++i)
            if (lane + 32 * i < dim) dst[lane + 32 * i] = x[i] * inv;
    } else if (unit < 2 * kv_heads + heads) {
        const int h = unit - 2 * kv_heads;
        for (int d = lane; d < vdim; d += 32)
            v[((size_t)t * heads + h) * vdim + d] = delta_conv(proj, proj_stride, kept, conv_w, conv_dtype, taps, channels, t, t0, 2 * qk + h * vdim + d);
    } else {
        const int h = unit - 2 * kv_heads - heads;
        const float rate = -expf(delta_weight(a_log, vec_dtype, h));
        for (int d = lane; d < dim; d += 32)
            lg[((size_t)t * heads + h) * dim + d] = rate * delta_softplus(raw[((size_t)t * heads + h) * dim + d] + delta_weight(dt_bias, vec_dtype, (size_t)h * dim + d));
        if (lane == 0) beta[(size_t)t * heads + h] = delta_sigmoid(proj[(size_t)t * proj_stride + channels + h]);
    }
}

// the last taps-1 inputs of every sequence after the step; a thread reads all it needs before it writes
__global__ void __launch_bounds__(256)
delta_conv_keep_kernel(const float* __restrict__ proj, int proj_stride, int taps, int channels, const int* __restrict__ seq_start,
                       const int* __restrict__ seq_slot, float* __restrict__ state, size_t state_stride) {
    chain_release();
    chain_wait();
    const int s = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int t0 = seq_start[s], t1 = seq_start[s + 1];
    float* kept = state + (size_t)seq_slot[s] * state_stride;
    float x[kDeltaMaxTaps];
    const int keep = taps - 1;
#pragma unroll
    for (int j = 0; j < kDeltaMaxTaps - 1; ++j)
        if (j < keep) {
            const int src = t1 - keep + j;
            x[j] = src >= t0 ? proj[(size_t)src * proj_stride + c] : kept[(size_t)(keep + (src - t0)) * channels + c];
        }
#pragma unroll
    for (int j = 0; j < kDeltaMaxTaps - 1; ++j)
        if (j < keep) kept[(size_t)j * channels + c] = x[j];
}

// the inner rows of the two low-rank projections in the compute dtype
__global__ void __launch_bounds__(128)
delta_inner_kernel(const float* __restrict__ proj, int proj_stride, int col, int decay_rank, int gate_rank, __nv_bfloat16* __restrict__ a,
                   int a_pitch, __nv_bfloat16* __restrict__ g, int g_pitch) {
    chain_release();
    chain_wait();
    const size_t t = blockIdx.x;
    const float* row = proj + t * proj_stride + col;
    for (int e = threadIdx.x; e < decay_rank + gate_rank; e += blockDim.x) {
        if (e < decay_rank) a[t * a_pitch + e] = __float2bfloat16_rn(row[e]);
        else g[t * g_pitch + e - decay_rank] = __float2bfloat16_rn(row[e]);
    }
}

// Block: 8 row groups (warps) x 32 columns; the thread of row group r keeps S[r + 8 i][c].  NR = ceil(dim / 8) at most.
constexpr int kScanGroups = 8, kScanCols = 32;
template <int NR>
__global__ void __launch_bounds__(kScanGroups * kScanCols)
delta_scan_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v,
                  const float* __restrict__ lg, const float* __restrict__ beta, const int* __restrict__ seq_start,
                  const int* __restrict__ seq_slot, float* __restrict__ state, size_t state_stride, float* __restrict__ out,
                  int heads, int kv_heads, int dim, int vdim) {
    chain_release();
    chain_wait();
    __shared__ float sq[kDeltaMaxDim], sk[kDeltaMaxDim], sg[kDeltaMaxDim];
    __shared__ float red[2][kScanGroups][kScanCols];
    const int s = blockIdx.x, h = blockIdx.y, c = blockIdx.z * kScanCols + (threadIdx.x & 31), r = threadIdx.x >> 5;
    const int t0 = seq_start[s], t1 = seq_start[s + 1];
    if (t1 <= t0) return;
    const int hk = h / (heads / kv_heads), lane = threadIdx.x & 31;
    const bool mine = c < vdim;
    float* st = state + (size_t)seq_slot[s] * state_stride + (size_t)h * dim * vdim;
    float S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = r + kScanGroups * i;
        S[i] = (mine && d < dim) ? st[(size_t)d * vdim + c] : 0.f;
    }
    for (int d = dim + threadIdx.x; d < kDeltaMaxDim; d += blockDim.x) { sq[d] = 0.f; sk[d] = 0.f; sg[d] = 0.f; }
    for (int t = t0; t < t1; ++t) {
        for (int d = threadIdx.x; d < dim; d += blockDim.x) {
            sq[d] = q[((size_t)t * kv_heads + hk) * dim + d];
            sk[d] = k[((size_t)t * kv_heads + hk) * dim + d];
            sg[d] = delta_decay(lg[((size_t)t * heads + h) * dim + d]);
        }
        const float b = beta[(size_t)t * heads + h];
        const float vc = mine ? v[((size_t)t * heads + h) * vdim + c] : 0.f;
        __syncthreads();
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            S[i] *= sg[r + kScanGroups * i];
            acc = fmaf(S[i], sk[r + kScanGroups * i], acc);
        }
        red[0][r][lane] = acc;
        __syncthreads();
        float seen = 0.f;
#pragma unroll
        for (int g = 0; g < kScanGroups; ++g) seen += red[0][g][lane];
        const float u = b * (vc - seen);
        acc = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            S[i] = fmaf(sk[r + kScanGroups * i], u, S[i]);
            acc = fmaf(S[i], sq[r + kScanGroups * i], acc);
        }
        red[1][r][lane] = acc;
        __syncthreads();
        if (r == 0 && mine) {
            float o = 0.f;
#pragma unroll
            for (int g = 0; g < kScanGroups; ++g) o += red[1][g][lane];
            out[((size_t)t * heads + h) * vdim + c] = o;
        }
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = r + kScanGroups * i;
        if (mine && d < dim) st[(size_t)d * vdim + c] = S[i];
    }
}

// ---------------------------------------------------------------- single tokens
// proj row of sequence s (or the sum of `splits` partial rows of row_width numbers): [q | k | v | b | a | g], floats.
// 512 threads: 512 / colsP row groups x colsP columns (v_dim rounded up to a multiple of 32); NR rows of S a thread at most.
constexpr int kTokThreads = 512;
static __host__ __device__ int tok_pitch(int rank) { return (rank * 2 + 127) / 128 * 64 + 32; }        // bfloat16 numbers of a staged row
static size_t tok_smem(int dim, int vdim, int decay_rank, int gate_rank) {
    const int colsP = (vdim + 31) / 32 * 32;
    return 2 * ((size_t)dim * tok_pitch(decay_rank) + (size_t)vdim * tok_pitch(gate_rank)) +
           sizeof(float) * (3 * (size_t)kDeltaMaxDim + 2 * (size_t)colsP + 2 * kTokThreads + decay_rank + gate_rank + 64);
}

template <int NR>
__global__ void __launch_bounds__(kTokThreads)
delta_token_kernel(const float* __restrict__ proj, int proj_stride, const float* __restrict__ partial, int splits, size_t split_stride,
                   int row_width, const __nv_bfloat16* __restrict__ a2, const __nv_bfloat16* __restrict__ g2, int decay_rank,
                   int gate_rank, const __nv_bfloat16* __restrict__ conv_w, int taps, const void* __restrict__ a_log,
                   const void* __restrict__ dt_bias, const void* __restrict__ norm_w, int vec_dtype, const int* __restrict__ seq_slot,
                   float* __restrict__ state, size_t state_stride, int conv_at, __nv_bfloat16* __restrict__ out, int heads, int dim,
                   int vdim, float unit_eps, float q_scale, float eps) {
    chain_release();
    extern __shared__ __align__(16) unsigned char tok_sm[];
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int colsP = (vdim + 31) & ~31, groups = kTokThreads / colsP;
    const int ap = tok_pitch(decay_rank), gp = tok_pitch(gate_rank);
    __nv_bfloat16* sa2 = reinterpret_cast<__nv_bfloat16*>(tok_sm);      // [dim][ap]
    __nv_bfloat16* sg2 = sa2 + (size_t)dim * ap;                         // [vdim][gp]
    float* sq = reinterpret_cast<float*>(sg2 + (size_t)vdim * gp);       // [256] each
    float* sk = sq + kDeltaMaxDim;
    float* sdec = sk + kDeltaMaxDim;
    float* sv = sdec + kDeltaMaxDim;                                     // [colsP]
    float* sgate = sv + colsP;                                           // [colsP]
    float* red = sgate + colsP;                                          // [2][512]
    float* inner = red + 2 * kTokThreads;                                // [decay_rank + gate_rank]
    float* small = inner + decay_rank + gate_rank;                       // [64]
    // the two small matrices' rows of this head: weights, asked for before the wait
    if (decay_rank % 8 == 0)
        for (int e = tid; e < dim * (decay_rank / 8); e += kTokThreads) {
            const int d = e / (decay_rank / 8), p = (e % (decay_rank / 8)) * 8;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"((uint32_t)__cvta_generic_to_shared(sa2 + (size_t)d * ap + p)),
                         "l"(a2 + ((size_t)h * dim + d) * decay_rank + p) : "memory");
        }
    else
        for (int e = tid; e < dim * decay_rank; e += kTokThreads) sa2[(size_t)(e / decay_rank) * ap + e % decay_rank] = a2[(size_t)h * dim * decay_rank + e];
    if (gate_rank % 8 == 0)
        for (int e = tid; e < vdim * (gate_rank / 8); e += kTokThreads) {
            const int d = e / (gate_rank / 8), p = (e % (gate_rank / 8)) * 8;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" :: "r"((uint32_t)__cvta_generic_to_shared(sg2 + (size_t)d * gp + p)),
                         "l"(g2 + ((size_t)h * vdim + d) * gate_rank + p) : "memory");
        }
    else
        for (int e = tid; e < vdim * gate_rank; e += kTokThreads) sg2[(size_t)(e / gate_rank) * gp + e % gate_rank] = g2[(size_t)h * vdim * gate_rank + e];
    asm volatile("cp.async.commit_group;" ::: "memory");
    chain_wait();
    const int c = tid % colsP, r = tid / colsP;
    const bool mine = c < vdim && r < groups;
    float* mem = state + (size_t)seq_slot[s] * state_stride;
    float* st = mem + (size_t)h * dim * vdim;
    float S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = r + groups * i;
        S[i] = (mine && d < dim) ? st[(size_t)d * vdim + c] : 0.f;
    }
    const float* prow = partial + (size_t)s * row_width;
    const float* row = proj + (size_t)s * proj_stride;
    auto input = [&](int col) {
        if (splits == 0) return row[col];
        float x = 0.f;
#pragma unroll 4
        for (int p = 0; p < splits; ++p) x += prow[(size_t)p * split_stride + col];
        return x;
    };
    const int qk = heads * dim, channels = 2 * qk + heads * vdim;
    float* kept = mem + conv_at;
    for (int e = tid; e < 2 * dim + vdim; e += kTokThreads) {            // convolutions of this head's channels
        const int ch = e < dim ? h * dim + e : e < 2 * dim ? qk + h * dim + e - dim : 2 * qk + h * vdim + e - 2 * dim;
        const float x = input(ch);
        float acc = to_float(conv_w[(size_t)ch * taps + taps - 1]) * x;
        float prev = x;                                                   // the kept inputs move up by one, newest last
        for (int j = taps - 2; j >= 0; --j) {
            const float old = kept[(size_t)j * channels + ch];
            acc = fmaf(to_float(conv_w[(size_t)ch * taps + j]), old, acc);
            kept[(size_t)j * channels + ch] = prev;
            prev = old;
        }
        const float y = delta_silu(acc);
        if (e < dim) sq[e] = y; else if (e < 2 * dim) sk[e - dim] = y; else sv[e - 2 * dim] = y;
    }
    for (int e = tid; e < decay_rank + gate_rank; e += kTokThreads) inner[e] = input(channels + heads + e);
    if (tid == kTokThreads - 1) small[0] = delta_sigmoid(input(channels + h));
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (warp < 2) {                                                       // unit vectors: factors of q and k
        const float* x = warp ? sk : sq;
        float acc = 0.f;
        for (int d = lane; d < dim; d += 32) acc = fmaf(x[d], x[d], acc);
        acc = warp_sum(acc);
        if (lane == 0) small[1 + warp] = (warp ? 1.0f : q_scale) / sqrtf(acc + unit_eps);
    }
    // four threads a row of the small matrices, eight numbers at a time
    for (int e = tid >> 2; e < ((dim + vdim + 7) & ~7); e += kTokThreads / 4) {
        const bool dec = e < dim;
        float acc = 0.f;
        if (e < dim + vdim) {
            const __nv_bfloat16* m = dec ? sa2 + (size_t)e * ap : sg2 + (size_t)(e - dim) * gp;
            const float* x = dec ? inner : inner + decay_rank;
            const int rank = dec ? decay_rank : gate_rank;
            for (int p = (tid & 3) * 8; p < rank; p += 32) {
                if (p + 8 <= rank) {
                    const uint4 raw = *reinterpret_cast<const uint4*>(m + p);
                    const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float2 f = __bfloat1622float2(b[i]);
                        acc = fmaf(f.x, x[p + 2 * i], acc);
                        acc = fmaf(f.y, x[p + 2 * i + 1], acc);
                    }
                } else {
                    for (int i = p; i < rank; ++i) acc = fmaf(to_float(m[i]), x[i], acc);
                }
            }
        }
        acc += __shfl_xor_sync(0xffffffffu, acc, 1);
        acc += __shfl_xor_sync(0xffffffffu, acc, 2);
        if ((tid & 3) == 0 && e < dim + vdim) {
            if (dec) sdec[e] = delta_decay(-expf(delta_weight(a_log, vec_dtype, h)) * delta_softplus(acc + delta_weight(dt_bias, vec_dtype, (size_t)h * dim + e)));
            else sgate[e - dim] = delta_sigmoid(acc);
        }
    }
    __syncthreads();
    const float b = small[0], fq = small[1], fk = small[2];
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = r + groups * i;
        if (d < dim) {
            S[i] *= sdec[d];
            acc = fmaf(S[i], sk[d], acc);
        }
    }
    red[tid] = acc;
    __syncthreads();
    float seen = 0.f;
    for (int g = 0; g < groups; ++g) seen += red[g * colsP + c];
    const float u = mine ? b * (sv[c] - seen * fk) : 0.f, uk = u * fk;
    acc = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = r + groups * i;
        if (d < dim) {
            S[i] = fmaf(sk[d], uk, S[i]);
            acc = fmaf(S[i], sq[d], acc);
            if (mine) st[(size_t)d * vdim + c] = S[i];
        }
    }
    red[kTokThreads + tid] = acc;
    __syncthreads();
    float o = 0.f;
    if (mine) {
        for (int g = 0; g < groups; ++g) o += red[kTokThreads + g * colsP + c];
        o *= fq;
    }
    // the norm over the head's columns: the first row group holds each once
    float sum = warp_sum(r == 0 ? o * o : 0.f);
    if (lane == 0) small[8 + warp] = sum;
    __syncthreads();
    sum = 0.f;
    for (int i = 0; i < colsP / 32; ++i) sum += small[8 + i];
    const float inv = 1.0f / sqrtf(sum / (float)vdim + eps);
    if (r == 0 && mine)
        out[((size_t)s * heads + h) * vdim + c] = __float2bfloat16_rn(o * inv * delta_weight(norm_w, vec_dtype, c) * sgate[c]);
}

static int tok_rows(int dim, int vdim) {
    const int colsP = (vdim + 31) / 32 * 32;
    if (colsP > kTokThreads) return 0;
    const int groups = kTokThreads / colsP, nr = (dim + groups - 1) / groups;
    return nr <= 8 ? 8 : nr <= 16 ? 16 : nr <= 32 ? 32 : 0;
}

// a warp per (row, head)
template <typename TG, typename TO>
__global__ void __launch_bounds__(256)
gated_head_rmsnorm_kernel(const float* __restrict__ o, const TG* __restrict__ gate, int gate_stride, const void* __restrict__ w,
                          int w_dtype, TO* __restrict__ out, int n_rows, int heads, int vdim, float eps, int gate_act, int w_heads,
                          float scale) {
    chain_release();
    chain_wait();
    const int pair = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (pair >= n_rows * heads) return;
    const int t = pair / heads, h = pair % heads;
    const float* row = o + (size_t)pair * vdim;
    float sq = 0.f;
    for (int d = lane; d < vdim; d += 32) sq = fmaf(row[d], row[d], sq);
    const float inv = scale / sqrtf(warp_sum(sq) / (float)vdim + eps);
    const int w0 = w_heads ? h * vdim : 0;
    for (int d = lane; d < vdim; d += 32) {
        const float g = to_float(gate[(size_t)t * gate_stride + h * vdim + d]);
        const float y = row[d] * inv * (w ? delta_weight(w, w_dtype, w0 + d) : 1.0f);
        out[(size_t)pair * vdim + d] = from_float<TO>(y * (gate_act ? delta_silu(g) : delta_sigmoid(g)));
    }
}

}  // namespace mdma

using namespace mdma;

extern "C" {

int mdma_delta_prepare(const float* proj, int proj_stride, const float* raw, const void* conv_w, int conv_dtype, int taps,
                       const void* a_log, const void* dt_bias, int vec_dtype, const int* tok_seq, const int* seq_start,
                       const int* seq_slot, const float* conv_state, long state_stride, float* q, float* k, float* v, float* lg,
                       float* beta, int n_rows, int heads, int kv_heads, int dim, int vdim, float unit_eps, float q_scale,
                       cudaStream_t stream) {
    MDMA_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0, "delta_prepare: bad sizes");
    MDMA_REQUIRE(dim <= kDeltaMaxDim, "delta_prepare: head size %d is beyond the limit %d", dim, kDeltaMaxDim);
    MDMA_REQUIRE(taps >= 1 && taps <= kDeltaMaxTaps, "delta_prepare: %d taps, the kernel takes 1..%d", taps, kDeltaMaxTaps);
    if (n_rows == 0) return 0;
    const int units = 2 * kv_heads + 2 * heads;
    launch_chained(delta_prepare_kernel, dim3(n_rows, (units + kDeltaPrepWarps - 1) / kDeltaPrepWarps), dim3(kDeltaPrepWarps * 32), 0,
                   stream, proj, proj_stride, raw, conv_w, conv_dtype, taps, a_log, dt_bias, vec_dtype, tok_seq, seq_start,
                   seq_slot, conv_state, (size_t)state_stride, q, k, v, lg, beta, heads, kv_heads, dim, vdim,
                   unit_eps, q_scale);
    MDMA_LAUNCH_OK("delta_prepare");
    return 0;
}

int mdma_delta_scan(const float* q, const float* k, const float* v, const float* lg, const float* beta, const int* seq_start,
                    const int* seq_slot, float* state, long state_stride, float* out, int n_seqs, int heads, int kv_heads,
                    int dim, int vdim, cudaStream_t stream) {
    MDMA_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0, "delta_scan: bad sizes");
    MDMA_REQUIRE(dim <= kDeltaMaxDim && heads <= 65535, "delta_scan: head size %d is beyond the limit %d", dim, kDeltaMaxDim);
    if (n_seqs == 0) return 0;
    dim3 grid(n_seqs, heads, (vdim + kScanCols - 1) / kScanCols);
#define MDMA_DELTA_SCAN(NR)                                                                                              \
    launch_chained(delta_scan_kernel<NR>, grid, dim3(kScanGroups * kScanCols), 0, stream, q, k, v, lg, beta, seq_start, seq_slot, \
                   state, (size_t)state_stride, out, heads, kv_heads, dim, vdim)
    if (dim <= 32) MDMA_DELTA_SCAN(4);
    else if (dim <= 64) MDMA_DELTA_SCAN(8);
    else if (dim <= 128) MDMA_DELTA_SCAN(16);
    else MDMA_DELTA_SCAN(32);
#undef MDMA_DELTA_SCAN
    MDMA_LAUNCH_OK("delta_scan");
    return 0;
}

// `gate_act` 0: sigmoid, 1: silu; `w` (vdim numbers, shared by the heads) may be null
int mdma_gated_head_rmsnorm(const float* o, const void* gate, int g_dtype, int gate_stride, const void* w, int w_dtype, void* out,
                            int out_dtype, int n_rows, int heads, int vdim, float eps, int gate_act, int w_heads, float scale,
                            cudaStream_t stream) {
    MDMA_REQUIRE(n_rows >= 0 && heads > 0 && vdim > 0, "gated_head_rmsnorm: bad sizes");
    if (n_rows == 0) return 0;
    const unsigned blocks = (unsigned)(((long)n_rows * heads + 7) / 8);
    MDMA_DISPATCH_DTYPE(g_dtype, TG, MDMA_DISPATCH_DTYPE(out_dtype, TO,
        launch_chained(gated_head_rmsnorm_kernel<TG, TO>, dim3(blocks), dim3(256), 0, stream, o, (const TG*)gate, gate_stride, w,
                       w_dtype, (TO*)out, n_rows, heads, vdim, eps, gate_act, w_heads, scale)));
    MDMA_LAUNCH_OK("gated_head_rmsnorm");
    return 0;
}

// Whether the single-token kernel takes these sizes.
int mdma_delta_token_fits(int heads, int kv_heads, int dim, int vdim, int decay_rank, int gate_rank, int taps) {
    return heads == kv_heads && dim <= kDeltaMaxDim && taps >= 1 && taps <= kDeltaMaxTaps && tok_rows(dim, vdim) > 0 &&
           tok_smem(dim, vdim, decay_rank, gate_rank) <= 200 * 1024;
}

// One token per sequence: proj rows [q | k | v | b | a | g] (or, with splits > 0, the sums of `splits` partial rows of
// row_width floats); a2 [heads * dim][decay_rank] and g2 [heads * vdim][gate_rank] bfloat16; a state row holds S, and from
// conv_at on the convolutions' kept inputs; out [sequences][heads * vdim] bfloat16.
int mdma_delta_token(const float* proj, int proj_stride, const float* partial, int splits, long split_stride, int row_width,
                     const void* a2, const void* g2, int decay_rank, int gate_rank, const void* conv_w, int taps, const void* a_log,
                     const void* dt_bias, const void* norm_w, int vec_dtype, const int* seq_slot, float* state, long state_stride,
                     int conv_at, void* out, int n_seqs, int heads, int dim, int vdim, float unit_eps, float q_scale, float eps,
                     cudaStream_t stream) {
    MDMA_REQUIRE(heads > 0 && dim > 0 && vdim > 0 && mdma_delta_token_fits(heads, heads, dim, vdim, decay_rank, gate_rank, taps),
                 "delta_token: heads of %d x %d are not a geometry this kernel takes", dim, vdim);
    MDMA_REQUIRE(splits >= 0 && (splits == 0 || partial) && heads <= 65535, "delta_token: bad arguments");
    MDMA_REQUIRE(row_width >= heads * (2 * dim + vdim + 1) + decay_rank + gate_rank, "delta_token: rows of %d numbers are too short", row_width);
    MDMA_REQUIRE((((uintptr_t)a2 | (uintptr_t)g2) & 15) == 0, "delta_token: matrices must start on 16 bytes");
    if (n_seqs == 0) return 0;
    const size_t smem = tok_smem(dim, vdim, decay_rank, gate_rank);
    const int nr = tok_rows(dim, vdim);
#define MDMA_TOK(NR)                                                                                                          \
    do {                                                                                                                      \
        static bool up = false;                                                                                               \
        if (!up) { cudaFuncSetAttribute(delta_token_kernel<NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); up = true; } \
        launch_chained(delta_token_kernel<NR>, dim3(n_seqs, heads), dim3(kTokThreads), smem, stream, proj, proj_stride, partial, splits, \
                       (size_t)split_stride, row_width, (const __nv_bfloat16*)a2, (const __nv_bfloat16*)g2, decay_rank, gate_rank, \
                       (const __nv_bfloat16*)conv_w, taps, a_log, dt_bias, norm_w, vec_dtype, seq_slot, state, (size_t)state_stride, \
                       conv_at, (__nv_bfloat16*)out, heads, dim, vdim, unit_eps, q_scale, eps);                               \
    } while (0)
    if (nr == 8) MDMA_TOK(8); else if (nr == 16) MDMA_TOK(16); else MDMA_TOK(32);
#undef MDMA_TOK
    MDMA_LAUNCH_OK("delta_token");
    return 0;
}

// a [rows][a_pitch] and g [rows][g_pitch] bfloat16 = columns [col, col + decay_rank) and the gate_rank after them
int mdma_delta_inner(const float* proj, int proj_stride, int col, int decay_rank, int gate_rank, void* a, int a_pitch, void* g,
                     int g_pitch, int n_rows, cudaStream_t stream) {
    if (n_rows == 0) return 0;
    launch_chained(delta_inner_kernel, dim3(n_rows), dim3(128), 0, stream, proj, proj_stride, col, decay_rank, gate_rank,
                   (__nv_bfloat16*)a, a_pitch, (__nv_bfloat16*)g, g_pitch);
    MDMA_LAUNCH_OK("delta_inner");
    return 0;
}

// The convolutions' kept inputs brought up to date after a step (columns [0, channels) of proj).
int mdma_delta_conv_keep(const float* proj, int proj_stride, int taps, int channels, const int* seq_start, const int* seq_slot,
                         float* conv_state, long state_stride, int n_seqs, cudaStream_t stream) {
    MDMA_REQUIRE(taps >= 1 && taps <= kDeltaMaxTaps && n_seqs <= 65535, "delta_conv_keep: %d taps, the kernel takes 1..%d", taps, kDeltaMaxTaps);
    if (n_seqs == 0 || taps == 1) return 0;
    launch_chained(delta_conv_keep_kernel, dim3((channels + 255) / 256, n_seqs), dim3(256), 0, stream, proj, proj_stride, taps,
                   channels, seq_start, seq_slot, conv_state, (size_t)state_stride);
    MDMA_LAUNCH_OK("delta_conv_keep");
    return 0;
}

}  // extern "C"
