// Attention whose heads' softmax weights are mixed before they meet the values.
//
// score_g(i, j) = factor_g (q_g . k_kv(g)), with a soft cap c > 0: c tanh(score / c); a query at position i sees key j if
// j <= i and (window 0, or i - j < window, or j < keep_first); w_g = softmax of head g over the visible keys;
// w'_h = sum_g M[h, g] w_g; the result of head h is sum_j w'_h(i, j) v_kv(h)(j).
//
// The visible keys of a row are numbered without the gap between the kept ones and the window: index e is position e
// below the gap and position e + gap above it.
//
// Kernel: a block per token, a warp per head, keys in that order 32 at a time, everything in float in one fixed order.
// First pass: every head's maximum and normaliser.  Second pass: the scores once more, the normalised weights of all
// heads for 32 keys into shared memory, every warp mixes its own row and adds the values of its own key/value head.
// The result of a token does not depend on the step's cut or on the batch.
#include "common.cuh"

namespace mdma {

constexpr int kMixMaxDim = 256, kMixMaxHeads = 32;

template <typename T>
__global__ void __launch_bounds__(kMixMaxHeads * 32)
mixed_weights_kernel(const T* __restrict__ q, int q_row_stride, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                     const float* __restrict__ mix, const float* __restrict__ factor, float softcap,
                     const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, const int* __restrict__ seq_slot,
                     const int* __restrict__ page_table, int max_pages, int page_size, T* __restrict__ out, int n_heads,
                     int n_kv_heads, int dim, int v_dim, int window, int keep_first) {
    chain_release();
    chain_wait();
    __shared__ float weights[kMixMaxHeads][33];
    const int t = blockIdx.x;
    const int h = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kvh = h / (n_heads / n_kv_heads);
    const int pos = tok_pos[t];
    const int first = window > 0 ? max(0, pos + 1 - window) : 0;
    const int kept = min(keep_first, first), gap = first - kept, n_keys = pos + 1 - gap;
    const int* pages = page_table + (size_t)seq_slot[tok_seq[t]] * max_pages;
    float qv[kMixMaxDim / 32], acc[kMixMaxDim / 32];
    const T* qp = q + (size_t)t * q_row_stride + (size_t)h * dim;
#pragma unroll
    for (int j = 0; j < kMixMaxDim / 32; ++j) {
        const int d = lane + 32 * j;
        qv[j] = d < dim ? to_float(qp[d]) : 0.f;
        acc[j] = 0.f;
    }
    const float f = factor[h];
    auto row_of = [&](int e) {
        const int p = e < kept ? e : e + gap;
        return ((size_t)pages[p / page_size] * page_size + (size_t)(p % page_size)) * n_kv_heads + kvh;
    };
    // lane k gets the score of key e0 + k
    auto scores = [&](int e0, int n) {
        float mine = -INFINITY;
        for (int k = 0; k < n; ++k) {
            const T* kp = k_cache + row_of(e0 + k) * dim;
            float part = 0.f;
#pragma unroll
            for (int j = 0; j < kMixMaxDim / 32; ++j) {
                const int d = lane + 32 * j;
                if (d < dim) part = fmaf(qv[j], to_float(kp[d]), part);
            }
            const float s = warp_sum(part) * f;
            if (lane == k) mine = softcap > 0.f ? softcap * tanhf(s / softcap) : s;
        }
        return mine;
    };
    float m = -INFINITY, l = 0.f;
    for (int e0 = 0; e0 < n_keys; e0 += 32) {
        const int n = min(32, n_keys - e0);
        const float s = scores(e0, n);
        const float m_new = fmaxf(m, warp_max(s));
        l = l * expf(m - m_new) + warp_sum(lane < n ? expf(s - m_new) : 0.f);
        m = m_new;
    }
    const float inv = 1.0f / l;
    for (int e0 = 0; e0 < n_keys; e0 += 32) {
        const int n = min(32, n_keys - e0);
        const float s = scores(e0, n);
        __syncthreads();                            // the mixing of the keys before has read `weights`
        weights[h][lane] = lane < n ? expf(s - m) * inv : 0.f;
        __syncthreads();
        float mixed = 0.f;
        for (int g = 0; g < n_heads; ++g) mixed = fmaf(mix[h * n_heads + g], weights[g][lane], mixed);
        for (int k = 0; k < n; ++k) {
            const T* vp = v_cache + row_of(e0 + k) * v_dim;
            const float w = __shfl_sync(0xffffffffu, mixed, k);
#pragma unroll
            for (int j = 0; j < kMixMaxDim / 32; ++j) {
                const int d = lane + 32 * j;
                if (d < v_dim) acc[j] = fmaf(w, to_float(vp[d]), acc[j]);
            }
        }
    }
    T* op = out + ((size_t)t * n_heads + h) * v_dim;
#pragma unroll
    for (int j = 0; j < kMixMaxDim / 32; ++j) {
        const int d = lane + 32 * j;
        if (d < v_dim) op[d] = from_float<T>(acc[j]);
    }
}

}  // namespace mdma

using namespace mdma;

extern "C" {

// mix [heads][heads]; factor [heads]: what a head's raw scores are multiplied by; softcap 0: none
int mdma_mixed_weights(const void* q, int dtype, int q_row_stride, const void* k_cache, const void* v_cache, const float* mix,
                       const float* factor, float softcap, const int* tok_seq, const int* tok_pos, const int* seq_slot,
                       const int* page_table, int max_pages, int page_size, void* out, int n_tokens, int n_heads,
                       int n_kv_heads, int dim, int v_dim, int window, int keep_first, cudaStream_t stream) {
    MDMA_REQUIRE(n_heads > 0 && n_heads <= kMixMaxHeads && n_kv_heads > 0 && n_heads % n_kv_heads == 0,
                 "mixed_weights: %d heads over %d kv heads (at most %d heads)", n_heads, n_kv_heads, kMixMaxHeads);
    MDMA_REQUIRE(dim > 0 && dim <= kMixMaxDim && v_dim > 0 && v_dim <= kMixMaxDim,
                 "mixed_weights: head sizes %d/%d are beyond the limit %d", dim, v_dim, kMixMaxDim);
    MDMA_REQUIRE(page_table && page_size > 0 && max_pages > 0 && window >= 0 && keep_first >= 0 && softcap >= 0.f && mix && factor,
                 "mixed_weights: bad arguments");
    if (n_tokens == 0) return 0;
    MDMA_DISPATCH_DTYPE(dtype, T,
        launch_chained(mixed_weights_kernel<T>, dim3(n_tokens), dim3(n_heads * 32), 0, stream, (const T*)q, q_row_stride,
                       (const T*)k_cache, (const T*)v_cache, mix, factor, softcap, tok_seq, tok_pos, seq_slot, page_table,
                       max_pages, page_size, (T*)out, n_heads, n_kv_heads, dim, v_dim, window, keep_first));
    MDMA_LAUNCH_OK("mixed_weights");
    return 0;
}

}  // extern "C"
