// Small kernels around attention and around a sublayer whose result is normed before it joins the residual stream.
//
// qk_prepare: a token's fused projection row [q heads | k heads | v heads | ...] is made ready for attention in one
// pass.  Every q and k head is rotated by the token's position (the first `rotary_dim` numbers of a head, pairs
// (2i, 2i+1) or (i, i + rotary_dim/2), angle = float(position) * inv_freq[i]) and then, if asked, divided by its own
// root mean square, x / sqrt(mean(x^2) + eps), without a weight.  q is written back in place; k and v go to the
// token's row of the paged cache (v heads may have a size of their own).  All arithmetic is float; a number is
// rounded once, when it is stored.
//
// head_gate: out[t, h, :] *= sigmoid(g[t, h]) * scale, one gate number per head (no gate: the scale alone).
//
// rmsnorm_add: x[t] += y[t] / sqrt(mean(y[t]^2) + eps) * w, the norm that follows a sublayer, in float.
#include "common.cuh"

namespace mdma {

constexpr int kPrepMaxDim = 256, kPrepWarps = 4;

template <typename T>
__global__ void __launch_bounds__(kPrepWarps * 32)
qk_prepare_kernel(T* __restrict__ proj, int row_stride, int k_col, int v_col, const int* __restrict__ tok_seq,
                  const int* __restrict__ tok_pos, const int* __restrict__ seq_slot, const float* __restrict__ inv_freq,
                  T* __restrict__ k_cache, T* __restrict__ v_cache, const int* __restrict__ page_table, int max_pages,
                  int page_size, int n_heads, int n_kv_heads, int dim, int v_dim, int rotary_dim, int interleaved,
                  int unit_norm, float eps, int write_kv) {
    chain_release();
    chain_wait();
    __shared__ float sines[kPrepMaxDim / 2], cosines[kPrepMaxDim / 2];
    __shared__ float rows[kPrepWarps][kPrepMaxDim];
    const int t = blockIdx.x;
    const int pos = tok_pos[t];
    const int half = rotary_dim / 2;
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)pos * inv_freq[i], &sines[i], &cosines[i]);
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int total = n_heads + (write_kv ? 2 * n_kv_heads : 0);
    const int head = blockIdx.y * kPrepWarps + warp;
    if (head >= total) return;
    T* row = proj + (size_t)t * row_stride;
    size_t cache_row = 0;
    if (write_kv) {
        const int slot = seq_slot[tok_seq[t]];
        cache_row = ((size_t)page_table[(size_t)slot * max_pages + pos / page_size] * page_size + (size_t)(pos % page_size)) * n_kv_heads;
    }
    if (head >= n_heads + n_kv_heads) {                 // a value head: copied as it is
        const int g = head - n_heads - n_kv_heads;
        const T* src = row + v_col + (size_t)g * v_dim;
        T* dst = v_cache + (cache_row + g) * v_dim;
        for (int d = lane; d < v_dim; d += 32) dst[d] = src[d];
        return;
    }
    const bool is_q = head < n_heads;
    T* src = is_q ? row + (size_t)head * dim : row + k_col + (size_t)(head - n_heads) * dim;
    T* dst = is_q ? src : k_cache + (cache_row + (head - n_heads)) * dim;
    float* v = rows[warp];
    for (int d = lane; d < dim; d += 32) v[d] = to_float(src[d]);
    __syncwarp();
    for (int i = lane; i < half; i += 32) {
        const int d0 = interleaved ? 2 * i : i, d1 = interleaved ? 2 * i + 1 : i + half;
        const float a = v[d0], b = v[d1], s = sines[i], c = cosines[i];
        v[d0] = a * c - b * s;
        v[d1] = b * c + a * s;
    }
    __syncwarp();
    float inv = 1.0f;
    if (unit_norm) {
        float sq = 0.f;
        for (int d = lane; d < dim; d += 32) sq = fmaf(v[d], v[d], sq);
        inv = 1.0f / sqrtf(warp_sum(sq) / (float)dim + eps);
    }
    for (int d = lane; d < dim; d += 32) dst[d] = from_float<T>(v[d] * inv);
}

template <typename T>
__global__ void __launch_bounds__(256)
head_gate_kernel(T* __restrict__ out, const T* __restrict__ gate, int gate_stride, int n_heads, int v_dim, float scale) {
    chain_release();
    chain_wait();
    const size_t t = blockIdx.x;
    const int width = n_heads * v_dim;
    for (int e = threadIdx.x; e < width; e += blockDim.x) {
        const float f = gate ? scale / (1.0f + expf(-to_float(gate[t * gate_stride + e / v_dim]))) : scale;
        out[t * width + e] = from_float<T>(to_float(out[t * width + e]) * f);
    }
}

// `partial` [splits][rows][width]: y is first completed by the partial sums a K-split product left (in split order), or
// with `only_partial` it is their sum.  `copy`: the new x in the compute dtype, for sublayers that read the stream itself.
template <typename TW, typename TC>
__global__ void __launch_bounds__(256)
rmsnorm_add_kernel(float* __restrict__ x, float* __restrict__ y, const float* __restrict__ partial, int splits,
                   size_t split_stride, int only_partial, const TW* __restrict__ w, int width, float eps, TC* __restrict__ copy) {
    chain_release();
    chain_wait();
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    float* yr = y + t * width;
    float sq = 0.f;
    for (int e = threadIdx.x; e < width; e += blockDim.x) {
        float v = only_partial ? 0.f : yr[e];
        for (int s = 0; s < splits; ++s) v += partial[(size_t)s * split_stride + t * width + e];
        if (splits > 0) yr[e] = v;
        sq = fmaf(v, v, sq);
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)width + eps);
    float* xr = x + t * width;
    for (int e = threadIdx.x; e < width; e += blockDim.x) {
        const float v = xr[e] + yr[e] * inv * to_float(w[e]);
        xr[e] = v;
        if (copy != nullptr) copy[t * width + e] = from_float<TC>(v);
    }
}

// The same, four columns a thread, the row in registers: rows of a multiple of four numbers, up to 4 NV a thread.  The
// partial sums of a number are asked for four at a time and added in split order.
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}
template <typename TW, typename TC, int NV>
__global__ void __launch_bounds__(512)
rmsnorm_add_vec_kernel(float* __restrict__ x, float* __restrict__ y, const float* __restrict__ partial, int splits,
                       size_t split_stride, int only_partial, const TW* __restrict__ w, int width, float eps, TC* __restrict__ copy) {
    chain_release();
    const int n4 = width >> 2;
    float4 wv[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {            // the weight is nobody's result: read before the wait
        const int e = threadIdx.x + k * blockDim.x;
        if (e < n4) wv[k] = make_float4(to_float(w[4 * e]), to_float(w[4 * e + 1]), to_float(w[4 * e + 2]), to_float(w[4 * e + 3]));
    }
    chain_wait();
    __shared__ float scratch[32];
    const size_t row = (size_t)blockIdx.x * width;
    float4 v[NV], xv[NV];
    float sq = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int e = threadIdx.x + k * blockDim.x;
        if (e < n4) {
            xv[k] = *reinterpret_cast<const float4*>(x + row + 4 * e);
            v[k] = only_partial ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(y + row + 4 * e);
            const float* p = partial + row + 4 * e;
#pragma unroll 4
            for (int s = 0; s < splits; ++s) {
                const float4 t = *reinterpret_cast<const float4*>(p + (size_t)s * split_stride);
                v[k].x += t.x; v[k].y += t.y; v[k].z += t.z; v[k].w += t.w;
            }
            if (splits > 0 && !only_partial) *reinterpret_cast<float4*>(y + row + 4 * e) = v[k];
            sq = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, fmaf(v[k].z, v[k].z, fmaf(v[k].w, v[k].w, sq))));
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)width + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int e = threadIdx.x + k * blockDim.x;
        if (e < n4) {
            const float4 r = make_float4(xv[k].x + v[k].x * inv * wv[k].x, xv[k].y + v[k].y * inv * wv[k].y,
                                         xv[k].z + v[k].z * inv * wv[k].z, xv[k].w + v[k].w * inv * wv[k].w);
            *reinterpret_cast<float4*>(x + row + 4 * e) = r;
            if (copy != nullptr) store4(copy + row + 4 * e, r);
        }
    }
}

// out = x in the compute dtype
__global__ void __launch_bounds__(256)
copy_rows_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ out, long n) {
    chain_release();
    chain_wait();
    for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long)gridDim.x * blockDim.x) out[i] = __float2bfloat16_rn(x[i]);
}

// y[t] += a * z[t]
__global__ void __launch_bounds__(256)
add_scaled_kernel(float* __restrict__ y, const float* __restrict__ z, float a, long n) {
    chain_release();
    chain_wait();
    for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long)gridDim.x * blockDim.x) y[i] = fmaf(a, z[i], y[i]);
}

}  // namespace mdma

using namespace mdma;

extern "C" {

int mdma_qk_prepare(void* proj, int dtype, int row_stride, int k_col, int v_col, const int* tok_seq, const int* tok_pos,
                    const int* seq_slot, const float* inv_freq, void* k_cache, void* v_cache, const int* page_table,
                    int max_pages, int page_size, int n_tokens, int n_heads, int n_kv_heads, int dim, int v_dim,
                    int rotary_dim, int interleaved, int unit_norm, float eps, int write_kv, cudaStream_t stream) {
    MDMA_REQUIRE(n_tokens >= 0 && n_heads > 0 && n_kv_heads >= 0, "qk_prepare: bad sizes");
    MDMA_REQUIRE(dim > 0 && dim <= kPrepMaxDim && v_dim > 0, "qk_prepare: head size %d is beyond the limit %d", dim, kPrepMaxDim);
    MDMA_REQUIRE(rotary_dim >= 0 && rotary_dim % 2 == 0 && rotary_dim <= dim, "qk_prepare: rotary_dim %d does not fit head size %d", rotary_dim, dim);
    MDMA_REQUIRE(rotary_dim == 0 || inv_freq, "qk_prepare: a rotation needs its frequencies");
    MDMA_REQUIRE(!write_kv || (page_table && k_cache && v_cache && page_size > 0 && max_pages > 0), "qk_prepare: no cache pages");
    if (n_tokens == 0) return 0;
    const int total = n_heads + (write_kv ? 2 * n_kv_heads : 0);
    MDMA_DISPATCH_DTYPE(dtype, T,
        launch_chained(qk_prepare_kernel<T>, dim3(n_tokens, (total + kPrepWarps - 1) / kPrepWarps), dim3(kPrepWarps * 32), 0,
                       stream, (T*)proj, row_stride, k_col, v_col, tok_seq, tok_pos, seq_slot, inv_freq, (T*)k_cache,
                       (T*)v_cache, page_table, max_pages, page_size, n_heads, n_kv_heads, dim, v_dim, rotary_dim,
                       interleaved, unit_norm, eps, write_kv));
    MDMA_LAUNCH_OK("qk_prepare");
    return 0;
}

int mdma_head_gate(void* out, const void* gate, int dtype, int gate_stride, int n_rows, int n_heads, int v_dim, float scale,
                   cudaStream_t stream) {
    MDMA_REQUIRE(n_rows >= 0 && n_heads > 0 && v_dim > 0, "head_gate: bad sizes");
    if (n_rows == 0) return 0;
    MDMA_DISPATCH_DTYPE(dtype, T,
        launch_chained(head_gate_kernel<T>, dim3(n_rows), dim3(256), 0, stream, (T*)out, (const T*)gate, gate_stride, n_heads,
                       v_dim, scale));
    MDMA_LAUNCH_OK("head_gate");
    return 0;
}

int mdma_rmsnorm_add(float* x, float* y, const float* partial, int splits, long split_stride, int only_partial, const void* w,
                     int w_dtype, int n_rows, int width, float eps, void* copy, int copy_dtype, cudaStream_t stream) {
    MDMA_REQUIRE(n_rows >= 0 && width > 0, "rmsnorm_add: bad sizes");
    MDMA_REQUIRE(splits >= 0 && (splits == 0 || partial), "rmsnorm_add: partial sums need a pointer");
    if (n_rows == 0) return 0;
    if (width % 4 == 0 && width <= 8192 && split_stride % 4 == 0 &&
        (((uintptr_t)x | (uintptr_t)y | (uintptr_t)partial | (uintptr_t)copy) & 15) == 0) {
        const int n4 = width / 4, threads = n4 >= 512 ? 512 : (n4 + 31) / 32 * 32, nv = (n4 + threads - 1) / threads;
#define MDMA_RA(NV)                                                                                                            \
        MDMA_DISPATCH_DTYPE(w_dtype, TW, MDMA_DISPATCH_DTYPE(copy_dtype, TC,                                                    \
            launch_chained(rmsnorm_add_vec_kernel<TW, TC, NV>, dim3(n_rows), dim3(threads), 0, stream, x, y, partial, \
                           splits, (size_t)split_stride, only_partial, (const TW*)w, width, eps, (TC*)copy)))
        if (nv == 1) MDMA_RA(1); else if (nv == 2) MDMA_RA(2); else MDMA_RA(4);
#undef MDMA_RA
        MDMA_LAUNCH_OK("rmsnorm_add");
        return 0;
    }
    MDMA_DISPATCH_DTYPE(w_dtype, TW, MDMA_DISPATCH_DTYPE(copy_dtype, TC,
        launch_chained(rmsnorm_add_kernel<TW, TC>, dim3(n_rows), dim3(256), 0, stream, x, y, partial, splits, (size_t)split_stride,
                       only_partial, (const TW*)w, width, eps, (TC*)copy)));
    MDMA_LAUNCH_OK("rmsnorm_add");
    return 0;
}

// out [n] bfloat16 = x [n]
int mdma_copy_rows(const float* x, void* out, long n, cudaStream_t stream) {
    if (n <= 0) return 0;
    long blocks = (n + 255) / 256;
    if (blocks > 1184) blocks = 1184;
    launch_chained(copy_rows_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, x, (__nv_bfloat16*)out, n);
    MDMA_LAUNCH_OK("copy_rows");
    return 0;
}

int mdma_add_scaled(float* y, const float* z, float a, long n, cudaStream_t stream) {
    if (n <= 0) return 0;
    long blocks = (n + 255) / 256;
    if (blocks > 1184) blocks = 1184;
    launch_chained(add_scaled_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, y, z, a, n);
    MDMA_LAUNCH_OK("add_scaled");
    return 0;
}

}  // extern "C"
