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

constexpr int kFinWarps = 8, kFinMaxDim = 256, kFinPerLane = kFinMaxDim / 32;

struct FinishParams {
    const void* rows;                  // finished rows (splits 0)
    const float* part_o; const float* part_ml; int splits;
    const float* sink_log2;
    int n_tokens, n_heads, maps, v_dim;
    float lambda, norm_scale, eps;     // two maps
    int gate_stride;
    float out_scale;
};

template <typename TI, typename TO>
__global__ void __launch_bounds__(kFinWarps * 32)
attention_finish_kernel(const FinishParams p, const TO* __restrict__ gate, TO* __restrict__ out) {
    chain_release();
    chain_wait();
    const int unit = blockIdx.x * kFinWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= p.n_tokens * p.n_heads) return;
    const int t = unit / p.n_heads, h = unit % p.n_heads;
    // a lane's numbers: quads 4 lane + 128 i where rows allow it, else lane + 32 i
    const bool quads = p.v_dim % 4 == 0;
    auto at = [&](int i) { return quads ? (i >> 2) * 128 + lane * 4 + (i & 3) : lane + 32 * i; };
    float o[kFinPerLane];
#pragma unroll
    for (int i = 0; i < kFinPerLane; ++i) o[i] = 0.f;
    for (int j = 0; j < p.maps; ++j) {
        const size_t row = (size_t)unit * p.maps + j;
        const float f = j == 0 ? 1.0f : -p.lambda;
        if (p.splits == 0) {
            const TI* src = reinterpret_cast<const TI*>(p.rows) + row * p.v_dim;
            if (quads && sizeof(TI) == 4) {
#pragma unroll
                for (int c = 0; c < kFinPerLane / 4; ++c)
                    if (at(4 * c) < p.v_dim) {
                        const float4 v = *reinterpret_cast<const float4*>(src + at(4 * c));
                        o[4 * c] = fmaf(f, v.x, o[4 * c]); o[4 * c + 1] = fmaf(f, v.y, o[4 * c + 1]);
                        o[4 * c + 2] = fmaf(f, v.z, o[4 * c + 2]); o[4 * c + 3] = fmaf(f, v.w, o[4 * c + 3]);
                    }
            } else {
#pragma unroll
                for (int i = 0; i < kFinPerLane; ++i)
                    if (at(i) < p.v_dim) o[i] = fmaf(f, to_float(src[at(i)]), o[i]);
            }
            continue;
        }
        const float* ml = p.part_ml + row * p.splits * 2;
        float m = -INFINITY, l = 0.f;
        for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ml[2 * s]);
        for (int s = 0; s < p.splits; ++s) if (ml[2 * s] != -INFINITY) l += exp2f(ml[2 * s] - m) * ml[2 * s + 1];
        if (p.sink_log2) l += exp2f(p.sink_log2[h] - m);
        float a[kFinPerLane];
#pragma unroll
        for (int i = 0; i < kFinPerLane; ++i) a[i] = 0.f;
        for (int s = 0; s < p.splits; ++s) {
            if (ml[2 * s] == -INFINITY) continue;                       // a run without a visible key
            const float w = exp2f(ml[2 * s] - m);
            const float* src = p.part_o + (row * p.splits + s) * p.v_dim;
#pragma unroll
            for (int i = 0; i < kFinPerLane; ++i)
                if (at(i) < p.v_dim) a[i] = fmaf(w, src[at(i)], a[i]);
        }
#pragma unroll
        for (int i = 0; i < kFinPerLane; ++i) o[i] = fmaf(f, a[i] / l, o[i]);
    }
    float scale = p.out_scale;
    if (p.maps > 1) {
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < kFinPerLane; ++i) sq = fmaf(o[i], o[i], sq);
        scale *= p.norm_scale / sqrtf(warp_sum(sq) / (float)p.v_dim + p.eps);
    }
    TO* dst = out + (size_t)unit * p.v_dim;
    const TO* g = gate ? gate + (size_t)t * p.gate_stride + (size_t)h * p.v_dim : nullptr;
#pragma unroll
    for (int i = 0; i < kFinPerLane; ++i) {
        if (at(i) >= p.v_dim) continue;
        float v = o[i] * scale;
        if (g) v *= 1.0f / (1.0f + expf(-to_float(g[at(i)])));
        dst[at(i)] = from_float<TO>(v);
    }
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
    MDMA_DISPATCH_DTYPE(rows_dtype, TI, MDMA_DISPATCH_DTYPE(out_dtype, TO,
        launch_chained(attention_finish_kernel<TI, TO>, dim3(blocks), dim3(kFinWarps * 32), 0, stream, p, (const TO*)gate, (TO*)out)));
    MDMA_LAUNCH_OK("attention_finish");
    return 0;
}

}  // extern "C"
