// What follows attention before its output product, a warp per (token, head):
//   - partial sums over runs of keys (`splits` > 1) are merged in order, a sink's exp joining the denominator once:
//         a_j = sum_s 2^(m_s - m) O_s / (sum_s 2^(m_s - m) l_s [+ 2^(sink - m)])
//     (splits 0: a_j are finished rows);
//   - two maps per head are taken apart: o = a_1 - lambda a_2, o <- o / sqrt(mean(o^2) + eps) * norm_scale over the
//     head's numbers (one map: o = a_1);
//   - o <- o * sigmoid(gate) * out_scale, element by element (no gate: the constant alone).
// Everything in float; rows [token][head][map][v_dim] in, [token][head][v_dim] out.
#include "common.cuh"

namespace mdma {

constexpr int kFinWarps = 8, kFinMaxDim = 256;

struct FinishParams {
    const void* rows;                  // finished rows (splits 0)
    const float* part_o; const float* part_ml; int splits;
    const float* sink_log2;
    int n_tokens, n_heads, maps, v_dim;
    float lambda, norm_scale, eps;     // two maps
    int gate_stride;
    float out_scale;
};

// four neighbouring numbers (the address is aligned to them)
__device__ __forceinline__ void fin_load4(const float* p, float* v) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void fin_load4(const __nv_bfloat16* p, float* v) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.y));
    v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
}
__device__ __forceinline__ void fin_store4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void fin_store4(__nv_bfloat16* p, const float* v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// VEC: heads of a multiple of four numbers, every row aligned to four; a lane owns the quads 4 lane + 128 i, else the
// numbers lane + 32 i.  NQ: quads a lane owns at most (1: heads up to 128).
template <typename TI, typename TO, bool VEC, int NQ>
__global__ void __launch_bounds__(kFinWarps * 32)
attention_finish_kernel(const FinishParams p, const TO* __restrict__ gate, TO* __restrict__ out) {
    chain_release();
    chain_wait();
    const int unit = blockIdx.x * kFinWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= p.n_tokens * p.n_heads) return;
    const int t = unit / p.n_heads, h = unit % p.n_heads;
    // f(number of the head, four of the lane's values at that place and how many of them are there)
    auto quads = [&](auto&& f) {
#pragma unroll
        for (int c = 0; c < NQ; ++c) {
            if (VEC) {
                const int d = c * 128 + lane * 4;
                if (d < p.v_dim) f(d, 4 * c, 4);
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int d = lane + 32 * (4 * c + i);
                    if (d < p.v_dim) f(d, 4 * c + i, 1);
                }
            }
        }
    };
    auto load = [](auto* src, float* v) {
        if constexpr (VEC) fin_load4(src, v);
        else v[0] = to_float(*src);
    };
    float o[4 * NQ];
#pragma unroll
    for (int i = 0; i < 4 * NQ; ++i) o[i] = 0.f;
    for (int j = 0; j < p.maps; ++j) {
        const size_t row = (size_t)unit * p.maps + j;
        const float f = j == 0 ? 1.0f : -p.lambda;
        if (p.splits == 0) {
            const TI* src = reinterpret_cast<const TI*>(p.rows) + row * p.v_dim;
            quads([&](int d, int i, int n) {
                float v[4];
                load(src + d, v);
#pragma unroll
                for (int e = 0; e < (VEC ? 4 : 1); ++e) o[i + e] = fmaf(f, v[e], o[i + e]);
            });
            continue;
        }
        const float* ml = p.part_ml + row * p.splits * 2;
        float m = -INFINITY, l = 0.f;
        for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ml[2 * s]);
        for (int s = 0; s < p.splits; ++s) if (ml[2 * s] != -INFINITY) l += exp2f(ml[2 * s] - m) * ml[2 * s + 1];
        if (p.sink_log2) l += exp2f(p.sink_log2[h] - m);
        const float share = f / l;
        float a[4 * NQ];
#pragma unroll
        for (int i = 0; i < 4 * NQ; ++i) a[i] = 0.f;
        for (int s = 0; s < p.splits; ++s) {
            if (ml[2 * s] == -INFINITY) continue;                       // a run without a visible key
            const float w = exp2f(ml[2 * s] - m);
            const float* src = p.part_o + (row * p.splits + s) * p.v_dim;
            quads([&](int d, int i, int n) {
                float v[4];
                load(src + d, v);
#pragma unroll
                for (int e = 0; e < (VEC ? 4 : 1); ++e) a[i + e] = fmaf(w, v[e], a[i + e]);
            });
        }
#pragma unroll
        for (int i = 0; i < 4 * NQ; ++i) o[i] = fmaf(share, a[i], o[i]);
    }
    float scale = p.out_scale;
    if (p.maps > 1) {
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < 4 * NQ; ++i) sq = fmaf(o[i], o[i], sq);
        scale *= p.norm_scale / sqrtf(warp_sum(sq) / (float)p.v_dim + p.eps);
    }
    TO* dst = out + (size_t)unit * p.v_dim;
    const TO* g = gate ? gate + (size_t)t * p.gate_stride + (size_t)h * p.v_dim : nullptr;
    quads([&](int d, int i, int n) {
        float v[4] = {1.f, 1.f, 1.f, 1.f};
        if (g) {
            load(g + d, v);
#pragma unroll
            for (int e = 0; e < (VEC ? 4 : 1); ++e) v[e] = 1.0f / (1.0f + expf(-v[e]));
        }
#pragma unroll
        for (int e = 0; e < (VEC ? 4 : 1); ++e) v[e] *= o[i + e] * scale;
        if constexpr (VEC) fin_store4(dst + d, v);
        else dst[d] = from_float<TO>(v[0]);
    });
}

}  // namespace mdma

using namespace mdma;

extern "C" {

// rows: finished rows in rows_dtype (splits 0), or part_o [..][splits][v_dim] and part_ml [..][splits][2]; maps 1 or 2.
int mdma_attention_finish(const void* rows, int rows_dtype, const float* part_o, const float* part_ml, int splits,
                          const float* sink_log2, const void* gate, int gate_stride, void* out, int out_dtype, int n_tokens,
                          int n_heads, int maps, int v_dim, float lambda, float norm_scale, float eps, float out_scale,
                          cudaStream_t stream) {
    MDMA_REQUIRE(n_tokens >= 0 && n_heads > 0 && (maps == 1 || maps == 2), "attention_finish: bad sizes");
    MDMA_REQUIRE(v_dim > 0 && v_dim <= kFinMaxDim, "attention_finish: value heads of %d are beyond the limit %d", v_dim, kFinMaxDim);
    MDMA_REQUIRE(splits >= 0 && (splits == 0 ? rows != nullptr : part_o && part_ml), "attention_finish: no rows");
    MDMA_REQUIRE(splits > 0 || rows_dtype != kF32 || ((uintptr_t)rows & 15) == 0, "attention_finish: float rows must be 16-byte aligned");
    if (n_tokens == 0) return 0;
    const FinishParams p = {rows, part_o, part_ml, splits, sink_log2, n_tokens, n_heads, maps, v_dim, lambda, norm_scale, eps, gate_stride, out_scale};
    const unsigned blocks = (unsigned)(((long)n_tokens * n_heads + kFinWarps - 1) / kFinWarps);
    const uintptr_t all = (uintptr_t)rows | (uintptr_t)part_o | (uintptr_t)out;
    const bool vec = v_dim % 4 == 0 && (all & 15) == 0 && ((uintptr_t)gate & (out_dtype == kF32 ? 15 : 7)) == 0 && (!gate || gate_stride % 4 == 0);
#define MDMA_FINISH(VEC, NQ)                                                                                                       \
    launch_chained(attention_finish_kernel<TI, TO, VEC, NQ>, dim3(blocks), dim3(kFinWarps * 32), 0, stream, p, (const TO*)gate, (TO*)out)
    MDMA_DISPATCH_DTYPE(rows_dtype, TI, MDMA_DISPATCH_DTYPE(out_dtype, TO, {
        if (!vec) MDMA_FINISH(false, 2);
        else if (v_dim <= 128) MDMA_FINISH(true, 1);
        else MDMA_FINISH(true, 2);
    }));
#undef MDMA_FINISH
    MDMA_LAUNCH_OK("attention_finish");
    return 0;
}

}  // extern "C"
