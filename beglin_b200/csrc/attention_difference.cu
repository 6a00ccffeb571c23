// The last step of differential attention behind the kernels that write partial results (attention.cu, attention_mma.cu):
// for every (row, head) the ranges of keys of BOTH maps are merged, the second map's result is taken off the first's, and the
// difference is normed.  With a_m = sum_s o_s e^(m_s - M) / sum_s l_s e^(m_s - M) over the splits s of map m,
//   o = a_1 - lambda a_2;   out[t, h, :] = o / sqrt(mean(o^2) + eps) * out_scale,
// all in float, rounded once when it is stored.  The partial results are those of 2 H heads (head h's maps are 2h and 2h + 1)
// of `hd` stored features, of which the first `vd` are the head's own.
//
// One CTA of eight warps per (row, head), four for each map.  Warp w of a map owns the splits s with s % 4 == w, in groups of
// sixteen consecutive ABSOLUTE split numbers: it asks for the four splits of its group at once and joins them in split order,
// and the four warps' results are joined in warp order.  So a row's result depends on nothing but its own range of splits.
#include "common.cuh"

namespace bg {

constexpr int DM_WARPS = 4;                 // per map
constexpr int DM_THREADS = 2 * DM_WARPS * 32;

template <typename TO, int DPL>
__global__ void __launch_bounds__(DM_THREADS)
difference_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, const int* __restrict__ positions,
                        TO* __restrict__ out, int out_stride, int H, int hd, int vd, int max_splits, int split_arg, int window,
                        float lambda, float out_scale, float eps) {
    __shared__ float acc_s[2 * DM_WARPS][32 * DPL];
    __shared__ float2 ml_s[2 * DM_WARPS];
    __shared__ float red[32];
    pdl_launch();
    const int t = blockIdx.x / H, h = blockIdx.x - t * H;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int map = warp / DM_WARPS, sub = warp % DM_WARPS;
    // (the row's position is written by no kernel of the step: its range of splits is worked out before the wait)
    const int pos = positions[t];
    const int split = keys_per_split(split_arg, pos + 1, max_splits);
    const int s_lo = first_visible(pos, window) / split, s_hi = pos / split;
    pdl_wait();
    const size_t prow = ((size_t)t * 2 * H + 2 * h + map) * max_splits;
    float m = -INFINITY, l = 0.0f, acc[DPL];
#pragma unroll
    for (int i = 0; i < DPL; ++i) acc[i] = 0.0f;
    for (int s0 = s_lo & ~15; s0 <= s_hi; s0 += 16) {
        float ms[4], ls[4], v[4][DPL];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int s = s0 + 4 * k + sub;
            const bool have = s >= s_lo && s <= s_hi;
            const float2 ml = have ? *reinterpret_cast<const float2*>(part_ml + (prow + s) * 2) : make_float2(-INFINITY, 0.0f);
            ms[k] = ml.x; ls[k] = ml.y;
#pragma unroll
            for (int i = 0; i < DPL; ++i) {
                const int d = i * 32 + lane;
                v[k][i] = (have && d < vd) ? part_o[(prow + s) * hd + d] : 0.0f;
            }
        }
        const float mg = fmaxf(fmaxf(ms[0], ms[1]), fmaxf(ms[2], ms[3]));
        if (mg == -INFINITY) continue;
        const float mn = fmaxf(m, mg);
        const float fo = (m == -INFINITY) ? 0.0f : expf(m - mn);
        l *= fo;
#pragma unroll
        for (int i = 0; i < DPL; ++i) acc[i] *= fo;
#pragma unroll
        for (int k = 0; k < 4; ++k) {                           // in split order
            if (ms[k] != -INFINITY) {
                const float f = expf(ms[k] - mn);
                l = fmaf(ls[k], f, l);
#pragma unroll
                for (int i = 0; i < DPL; ++i) acc[i] = fmaf(v[k][i], f, acc[i]);
            }
        }
        m = mn;
    }
#pragma unroll
    for (int i = 0; i < DPL; ++i) acc_s[warp][i * 32 + lane] = acc[i];
    if (lane == 0) ml_s[warp] = make_float2(m, l);
    __syncthreads();
    // a thread per feature: the four warps of each map in warp order, then the difference
    const int d = threadIdx.x;
    float o = 0.0f;
    if (d < vd) {
        float a[2];
#pragma unroll
        for (int c = 0; c < 2; ++c) {
            float mt = -INFINITY;
#pragma unroll
            for (int w = 0; w < DM_WARPS; ++w) mt = fmaxf(mt, ml_s[c * DM_WARPS + w].x);
            float lt = 0.0f, at = 0.0f;
#pragma unroll
            for (int w = 0; w < DM_WARPS; ++w) {
                const float2 ml = ml_s[c * DM_WARPS + w];
                const float f = (ml.x == -INFINITY) ? 0.0f : expf(ml.x - mt);
                lt = fmaf(ml.y, f, lt);
                at = fmaf(acc_s[c * DM_WARPS + w][d], f, at);
            }
            a[c] = at / lt;
        }
        o = a[0] - lambda * a[1];
    }
    const float ss = block_sum(o * o, red);
    const float mult = out_scale / sqrtf(ss / (float)vd + eps);
    if (d < vd) out[(size_t)t * out_stride + (size_t)h * vd + d] = from_float<TO>(o * mult);
}

}  // namespace bg

using namespace bg;

// part_o [T * 2 H][max_splits][hd], part_ml [T * 2 H][max_splits][2]; out [T][H * vd]; vd <= 256.
extern "C" int bg_difference_merge(const float* part_o, const float* part_ml, const int* positions, void* out, int out_dtype,
                                   int out_stride, int T, int H, int hd, int vd, int max_splits, int split, int window,
                                   float lambda, float out_scale, float eps, cudaStream_t stream) {
    if (T <= 0 || H <= 0) return BG_OK;
    if (vd <= 0 || vd > hd || vd > DM_THREADS || max_splits < 1 || (long long)T * H > 0x7fffffffLL) return BG_ERR_SHAPE;
    BG_DISPATCH_DTYPE(out_dtype, TO, {
        if (vd <= 128) launch(difference_merge_kernel<TO, 4>, dim3(T * H), dim3(DM_THREADS), 0, stream, part_o, part_ml, positions, (TO*)out, out_stride, H, hd, vd, max_splits, split, window, lambda, out_scale, eps);
        else launch(difference_merge_kernel<TO, 8>, dim3(T * H), dim3(DM_THREADS), 0, stream, part_o, part_ml, positions, (TO*)out, out_stride, H, hd, vd, max_splits, split, window, lambda, out_scale, eps);
    });
    BG_LAUNCH_CHECK();
    return BG_OK;
}
