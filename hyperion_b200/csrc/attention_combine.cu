// What follows the two softmax maps of a differential attention head, in one launch: the pieces of the keys each map's attention was split
// into are put together (or, where a map's result is whole, taken as it is), and then, per token and head,
//     o = a1 - lambda a2;   o <- o / sqrt(mean(o^2) + eps) * post;   out = o * sigmoid(gate)
// entry by entry over the head's values.  Everything is float until the one rounding at the store.  A warp serves a (token, head), so the
// sum of squares has one shape whatever else is in the launch.
#include "common.cuh"

namespace {
constexpr int WARPS = 4;

// pieces [items, heads, 2, splits, v_dim] float with (maximum in the exp2 domain, sum) per piece in ml, or, without ml, results
// [tokens, heads, 2, v_dim] (splits 1).  items: the token of an item, or null (item i is token i).
template <typename TO, int PER_LANE>
__global__ void __launch_bounds__(32 * WARPS) differential_combine_kernel(const float* __restrict__ pieces, const float2* __restrict__ ml, const int* __restrict__ items,
                                                                          int heads, int splits, int v_dim, float lambda, float eps, float post,
                                                                          const float* __restrict__ gate, int gate_stride, int gate_off, TO* __restrict__ out,
                                                                          int out_stride) {
    const int item = blockIdx.x, head = blockIdx.y * WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    let_next_kernel_start();
    wait_for_previous_kernels();
    if (head >= heads) return;
    const int t = items ? items[item] : item;
    float o[PER_LANE], gated[PER_LANE];
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
        const int c = lane + 32 * i;
        gated[i] = c < v_dim ? gate[(size_t)t * gate_stride + gate_off + (size_t)head * v_dim + c] : 0.f;
    }
#pragma unroll
    for (int map = 0; map < 2; ++map) {
        const size_t slot0 = (((size_t)item * heads + head) * 2 + map) * splits;
        float a[PER_LANE];
        if (!ml) {
#pragma unroll
            for (int i = 0; i < PER_LANE; ++i) {
                const int c = lane + 32 * i;
                a[i] = c < v_dim ? pieces[slot0 * v_dim + c] : 0.f;
            }
        } else {
            float m = -INFINITY, l = 0.f;
            for (int s = 0; s < splits; ++s) m = fmaxf(m, ml[slot0 + s].x);
#pragma unroll
            for (int i = 0; i < PER_LANE; ++i) a[i] = 0.f;
#pragma unroll 4
            for (int s = 0; s < splits; ++s) {
                const float2 p = ml[slot0 + s];
                const float f = p.x == -INFINITY ? 0.f : exp2f(p.x - m);
                l = fmaf(f, p.y, l);
#pragma unroll
                for (int i = 0; i < PER_LANE; ++i) {
                    const int c = lane + 32 * i;
                    if (c < v_dim) a[i] = fmaf(f, pieces[(slot0 + s) * v_dim + c], a[i]);
                }
            }
            const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
            for (int i = 0; i < PER_LANE; ++i) a[i] *= inv;
        }
#pragma unroll
        for (int i = 0; i < PER_LANE; ++i) o[i] = map == 0 ? a[i] : fmaf(-lambda, a[i], o[i]);
    }
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) sum = fmaf(o[i], o[i], sum);
    const float scale = post / sqrtf(warp_sum(sum) / (float)v_dim + eps);
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
        const int c = lane + 32 * i;
        if (c < v_dim) out[(size_t)t * out_stride + (size_t)head * v_dim + c] = from_float<TO>(o[i] * scale / (1.f + expf(-gated[i])));
    }
}
}  // namespace

HB_EXPORT int hb_differential_combine(const float* pieces, const float* ml, const int* items, int n_items, int heads, int splits, int v_dim, float lambda, float eps,
                                      float post, const float* gate, int gate_stride, int gate_off, void* out, int out_stride, int out_is_bf16,
                                      cudaStream_t stream) {
    if (n_items <= 0) return 0;
    if (!pieces || !gate || !out || heads <= 0 || splits < 1 || (splits > 1 && !ml)) return HB_BAD_ARGUMENT;
    if (v_dim <= 0 || v_dim > 640 || heads > 65535 * WARPS) return HB_UNSUPPORTED_SIZE;
    const dim3 grid(n_items, (heads + WARPS - 1) / WARPS);
#define HB_COMBINE(TO, N)                                                                                                                                   \
    return launch_after_previous(differential_combine_kernel<TO, N>, grid, dim3(32 * WARPS), 0, stream, pieces, (const float2*)ml, items, heads, splits, v_dim, \
                                 lambda, eps, post, gate, gate_stride, gate_off, (TO*)out, out_stride)
    if (out_is_bf16) {
        if (v_dim <= 128) HB_COMBINE(__nv_bfloat16, 4);
        if (v_dim <= 256) HB_COMBINE(__nv_bfloat16, 8);
        HB_COMBINE(__nv_bfloat16, 20);
    }
    if (v_dim <= 128) HB_COMBINE(float, 4);
    if (v_dim <= 256) HB_COMBINE(float, 8);
    HB_COMBINE(float, 20);
#undef HB_COMBINE
}
