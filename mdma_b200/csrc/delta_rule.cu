// The gated delta rule with a decay per key channel, and the gated norm per head that follows it.
//
// Per head, with unit vectors q (times dim^-1/2) and k [dim], v [vdim], a step size b and decays g [dim] of a token:
//     S <- diag(g) S;   u = b (v - S^T k);   S <- S + k u^T;   o = S^T q          S [dim][vdim] floats per sequence
//
// delta_prepare: from the projections to what enters the recurrence, all in float, a warp per (token, unit): q and k
// heads pass a short causal convolution per channel and silu and become unit vectors, v heads pass convolution and
// silu, decay heads become log g = -exp(A_log) softplus(a + dt_bias), and b = sigmoid(its logit).
//
// delta_scan: row by row, block = (sequence, head, 32 columns of S).  Every thread keeps its part of S in registers for
// all rows of the step; every sum has one fixed order, so the result does not depend on how rows were cut into steps.
// The 32-bit engine's walk, short portions and, with the preparation inside, single tokens.
//
// gated_head_rmsnorm: out = o_h / sqrt(mean(o_h^2) + eps) [* w] * act(gate), per head, act = sigmoid or silu.
#include "common.cuh"

namespace mdma {

constexpr int kDeltaMaxDim = 256, kDeltaMaxTaps = 16;

__device__ __forceinline__ float delta_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float delta_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float delta_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// exp(x), x <= 0, rounded once where it lies near one: a slow channel's decays are multiplied over thousands of tokens,
// and an error of a unit in the last place to one side would add up over them
__device__ __forceinline__ float delta_decay(float x) { return x > -0.5f ? 1.0f + expm1f(x) : expf(x); }
__device__ __forceinline__ float delta_weight(const void* w, int dtype, size_t e) {
    return dtype == kF32 ? reinterpret_cast<const float*>(w)[e] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(w)[e]);
}

// silu of the short convolution of channel c at row t (proj rows hold the inputs at column c; rows before the step's
// first row t0 come from the kept inputs)
__device__ __forceinline__ float delta_conv(const float* __restrict__ proj, int stride, const float* __restrict__ kept,
                                            const void* __restrict__ w, int w_dtype, int taps, int channels, int t, int t0, int c) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int src = t - (taps - 1) + j;
        const float x = src >= t0 ? proj[(size_t)src * stride + c] : kept[(size_t)(taps - 1 + (src - t0)) * channels + c];
        acc = fmaf(delta_weight(w, w_dtype, (size_t)c * taps + j), x, acc);
    }
    return delta_silu(acc);
}

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

// a warp per (row, head)
template <typename TG, typename TO>
__global__ void __launch_bounds__(256)
gated_head_rmsnorm_kernel(const float* __restrict__ o, const TG* __restrict__ gate, int gate_stride, const void* __restrict__ w,
                          int w_dtype, TO* __restrict__ out, int n_rows, int heads, int vdim, float eps, int gate_act) {
    chain_release();
    chain_wait();
    const int pair = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (pair >= n_rows * heads) return;
    const int t = pair / heads, h = pair % heads;
    const float* row = o + (size_t)pair * vdim;
    float sq = 0.f;
    for (int d = lane; d < vdim; d += 32) sq = fmaf(row[d], row[d], sq);
    const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)vdim + eps);
    for (int d = lane; d < vdim; d += 32) {
        const float g = to_float(gate[(size_t)t * gate_stride + h * vdim + d]);
        const float y = row[d] * inv * (w ? delta_weight(w, w_dtype, d) : 1.0f);
        out[(size_t)pair * vdim + d] = from_float<TO>(y * (gate_act ? delta_silu(g) : delta_sigmoid(g)));
    }
}

}  // namespace mdma

using namespace mdma;

extern "C" {

int mdma_delta_prepare(const float* proj, int proj_stride, const float* raw, const void* conv_w, int conv_dtype, int taps,
                       const void* a_log, const void* dt_bias, int vec_dtype, const int* tok_seq, const int* seq_start,
                       const int* seq_slot, float* conv_state, long state_stride, float* q, float* k, float* v, float* lg,
                       float* beta, int n_rows, int n_seqs, int heads, int kv_heads, int dim, int vdim, float unit_eps,
                       float q_scale, cudaStream_t stream) {
    MDMA_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0, "delta_prepare: bad sizes");
    MDMA_REQUIRE(dim <= kDeltaMaxDim, "delta_prepare: head size %d is beyond the limit %d", dim, kDeltaMaxDim);
    MDMA_REQUIRE(taps >= 1 && taps <= kDeltaMaxTaps, "delta_prepare: %d taps, the kernel takes 1..%d", taps, kDeltaMaxTaps);
    MDMA_REQUIRE(n_seqs <= 65535, "delta_prepare: too many sequences");
    if (n_rows == 0) return 0;
    const int units = 2 * kv_heads + 2 * heads, channels = 2 * kv_heads * dim + heads * vdim;
    launch_chained(delta_prepare_kernel, dim3(n_rows, (units + kDeltaPrepWarps - 1) / kDeltaPrepWarps), dim3(kDeltaPrepWarps * 32), 0,
                   stream, proj, proj_stride, raw, conv_w, conv_dtype, taps, a_log, dt_bias, vec_dtype, tok_seq, seq_start,
                   seq_slot, (const float*)conv_state, (size_t)state_stride, q, k, v, lg, beta, heads, kv_heads, dim, vdim,
                   unit_eps, q_scale);
    MDMA_LAUNCH_OK("delta_prepare");
    if (taps > 1) {
        launch_chained(delta_conv_keep_kernel, dim3((channels + 255) / 256, n_seqs), dim3(256), 0, stream, proj, proj_stride, taps,
                       channels, seq_start, seq_slot, conv_state, (size_t)state_stride);
        MDMA_LAUNCH_OK("delta_conv_keep");
    }
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
                            int out_dtype, int n_rows, int heads, int vdim, float eps, int gate_act, cudaStream_t stream) {
    MDMA_REQUIRE(n_rows >= 0 && heads > 0 && vdim > 0, "gated_head_rmsnorm: bad sizes");
    if (n_rows == 0) return 0;
    const unsigned blocks = (unsigned)(((long)n_rows * heads + 7) / 8);
    MDMA_DISPATCH_DTYPE(g_dtype, TG, MDMA_DISPATCH_DTYPE(out_dtype, TO,
        launch_chained(gated_head_rmsnorm_kernel<TG, TO>, dim3(blocks), dim3(256), 0, stream, o, (const TG*)gate, gate_stride, w,
                       w_dtype, (TO*)out, n_rows, heads, vdim, eps, gate_act)));
    MDMA_LAUNCH_OK("gated_head_rmsnorm");
    return 0;
}

}  // extern "C"
