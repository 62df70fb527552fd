// Several residual streams instead of one.  A sublayer f reads one mixture of the streams x_0 .. x_(S-1) and writes to all of them:
//     u = sum_s read[s] x_s;   y = f(norm(u));   x_t <- sum_s mix[s, t] x_s + share[t] y   (every new stream from the old ones)
// One launch per sublayer boundary does what lies between a sublayer's last product and the next one's first: the sublayer's result
// joins the streams, the next sublayer's mixture is taken from the new streams, divided by its root mean square and multiplied by the norm's
// weight.  The result may be one tensor, or the sum of two, each first divided by its own root mean square and multiplied by its
// own weight, the sum times a factor (two mixers side by side); either may still lie in split-K pieces, which are added up in split
// order.  Where the streams are still all equal (the start of a model) one row per token stands for all of them.  A column never
// meets another one but in the sums of squares, so a thread owns its columns of all streams and works in place.  Everything is float
// until the one rounding of the normalised row; a row's sums have one shape for a given width, whatever else is in the launch.
// Built once per number of streams: HB_STREAMS is 1 to 4, or 0 for a kernel that takes any number up to 16.
#include "common.cuh"

#ifndef HB_STREAMS
#define HB_STREAMS 0
#endif

namespace {
struct HyperArgs {
    const float* src;       // [tokens, streams, hidden], or [tokens, hidden] when `single`
    int single;
    float* dst;             // where the new streams go ([tokens, streams, hidden]; may be src), or null: nobody reads them
    int streams;
    const void* y[2];       // the sublayer's result(s) [tokens, hidden]; float [splits, tokens, hidden] where splits > 0; y[1] may be null
    int splits[2];
    size_t split_stride;
    const float* y_norm[2]; // a norm on each result (null: as it is)
    float y_eps, y_scale;
    const float* mix;       // [streams, streams] from, to; null: nothing is pending, the streams stay as they are
    const float* share;     // [streams]
    const float* read;      // [streams]; null: the sum of the streams
    const float* weight;    // [hidden]: the next norm
    float eps;
    void* out;              // [rows, hidden]
    const int* rows;        // the rows to work on, or null: all of them
    int hidden;
};

template <typename T, int VEC>
__device__ __forceinline__ void take(const T* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) load4(p, v);
    else v[0] = to_float(p[0]);
}

template <typename T, int VEC>
__device__ __forceinline__ void put(T* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) store4(p, v);
    else p[0] = from_float<T>(v[0]);
}

template <typename TD, int VEC>
__device__ __forceinline__ void take_result(const HyperArgs& a, int which, size_t at, float (&v)[VEC]) {
    if (a.splits[which] > 0) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = 0.f;
        const float* p = (const float*)a.y[which] + at;
        float piece[VEC];
#pragma unroll 8
        for (int k = 0; k < a.splits[which]; ++k) {
            take<float, VEC>(p + (size_t)k * a.split_stride, piece);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] += piece[e];
        }
    } else {
        take<TD, VEC>((const TD*)a.y[which] + at, v);
    }
}

// SMAX: the streams, or (HB_STREAMS 0) the most of them.
template <typename TD, typename TO, int VEC, int CHUNKS, int SMAX>
__global__ void __launch_bounds__(512, CHUNKS <= 2 && SMAX <= 4 ? 2 : 1) hyper_connect_kernel(const HyperArgs a) {
    constexpr bool EXACT = HB_STREAMS > 0, AHEAD = EXACT && CHUNKS == 1;  // a row's streams are asked for before the sums of squares (more of them cost a block of occupancy)
    __shared__ float scratch[32];
    const int r = blockIdx.x, step = blockDim.x * VEC, hidden = a.hidden;
    const int streams = EXACT ? SMAX : a.streams;
    __shared__ __align__(16) float mix[EXACT ? SMAX : 1][EXACT ? SMAX : 1], share[EXACT ? SMAX : 1], read[EXACT ? SMAX : 1];  // mix[t][s]: from s to t
    let_next_kernel_start();
    if constexpr (EXACT) {  // no kernel writes weights: these loads overlap the kernel before
        if (threadIdx.x < SMAX * SMAX) {
            const int t = threadIdx.x / SMAX, s = threadIdx.x % SMAX;
            mix[t][s] = a.mix ? a.mix[s * SMAX + t] : (s == t ? 1.f : 0.f);
        }
        if (threadIdx.x < SMAX) {
            read[threadIdx.x] = a.read ? a.read[threadIdx.x] : 1.f;
            share[threadIdx.x] = a.mix ? a.share[threadIdx.x] : 0.f;
        }
        __syncthreads();
    }
    wait_for_previous_kernels();
    const int row = a.rows ? a.rows[r] : r;
    const float* src = a.src + (size_t)row * hidden * (a.single ? 1 : streams);
    float* dst = a.dst ? a.dst + (size_t)row * hidden * streams : nullptr;
    const size_t stream_stride = a.single ? 0 : (size_t)hidden;

    float kept[AHEAD ? CHUNKS : 1][AHEAD ? SMAX : 1][VEC];
    float y[CHUNKS][VEC];
    if (a.mix) {
        float y2[CHUNKS][VEC], sum0 = 0.f, sum1 = 0.f;
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int i = c * step + threadIdx.x * VEC;
            if (i >= hidden) continue;
            take_result<TD, VEC>(a, 0, (size_t)row * hidden + i, y[c]);
            if (a.y[1]) take_result<TD, VEC>(a, 1, (size_t)row * hidden + i, y2[c]);
        }
        if constexpr (AHEAD) {
#pragma unroll
            for (int c = 0; c < CHUNKS; ++c) {
                const int i = c * step + threadIdx.x * VEC;
                if (i >= hidden) continue;
#pragma unroll
                for (int s = 0; s < SMAX; ++s) take<float, VEC>(src + (size_t)s * stream_stride + i, kept[c][s]);
            }
        }
        float inv0 = a.y_scale, inv1 = a.y_scale;
        if (a.y_norm[0] || a.y_norm[1]) {
#pragma unroll
            for (int c = 0; c < CHUNKS; ++c) {
                const int i = c * step + threadIdx.x * VEC;
                if (i >= hidden) continue;
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    sum0 = fmaf(y[c][e], y[c][e], sum0);
                    if (a.y[1]) sum1 = fmaf(y2[c][e], y2[c][e], sum1);
                }
            }
            if (a.y_norm[0]) inv0 *= 1.0f / sqrtf(block_sum(sum0, scratch) / (float)hidden + a.y_eps);
            if (a.y[1] && a.y_norm[1]) inv1 *= 1.0f / sqrtf(block_sum(sum1, scratch) / (float)hidden + a.y_eps);
        }
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) {
            const int i = c * step + threadIdx.x * VEC;
            if (i >= hidden) continue;
            float w[VEC];
            if (a.y_norm[0]) {
                take<float, VEC>(a.y_norm[0] + i, w);
#pragma unroll
                for (int e = 0; e < VEC; ++e) y[c][e] *= w[e];
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) y[c][e] *= inv0;
            if (a.y[1]) {
                if (a.y_norm[1]) {
                    take<float, VEC>(a.y_norm[1] + i, w);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) y2[c][e] *= w[e];
                }
#pragma unroll
                for (int e = 0; e < VEC; ++e) y[c][e] = fmaf(y2[c][e], inv1, y[c][e]);
            }
        }
    }
    float sum = 0.f;
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {  // from here on y holds the mixture that the next sublayer reads
        const int i = c * step + threadIdx.x * VEC;
        if (i >= hidden) continue;
        float x[SMAX][VEC], u[VEC];
#pragma unroll
        for (int s = 0; s < SMAX; ++s) {
            if (s >= streams) continue;
            if (AHEAD && a.mix) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) x[s][e] = kept[AHEAD ? c : 0][AHEAD ? s : 0][e];
            } else {
                take<float, VEC>(src + (size_t)s * stream_stride + i, x[s]);
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] = 0.f;
#pragma unroll
        for (int t = 0; t < SMAX; ++t) {
            if (t >= streams) continue;
            float now[VEC];
            if (a.mix) {
                const float part = EXACT ? share[EXACT ? t : 0] : a.share[t];
#pragma unroll
                for (int e = 0; e < VEC; ++e) now[e] = 0.f;
#pragma unroll
                for (int s = 0; s < SMAX; ++s) {
                    if (s >= streams) continue;
                    const float m = EXACT ? mix[EXACT ? t : 0][EXACT ? s : 0] : a.mix[s * streams + t];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) now[e] = fmaf(m, x[s][e], now[e]);
                }
#pragma unroll
                for (int e = 0; e < VEC; ++e) now[e] = fmaf(part, y[c][e], now[e]);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) now[e] = x[t][e];
            }
            if (dst) put<float, VEC>(dst + (size_t)t * hidden + i, now);
            const float weight = EXACT ? read[EXACT ? t : 0] : (a.read ? a.read[t] : 1.f);
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[e] = fmaf(weight, now[e], u[e]);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            y[c][e] = u[e];
            sum = fmaf(u[e], u[e], sum);
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + a.eps);
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = c * step + threadIdx.x * VEC;
        if (i >= hidden) continue;
        float w[VEC];
        take<float, VEC>(a.weight + i, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[c][e] *= inv * w[e];
        put<TO, VEC>((TO*)a.out + (size_t)r * hidden + i, y[c]);
    }
}

template <typename TD, typename TO>
int launch_streams(const HyperArgs& a, int n_rows, bool by_four, int threads, int chunks, cudaStream_t stream) {
#define HB_HYPER(VEC, CHUNKS) return launch_after_previous(hyper_connect_kernel<TD, TO, VEC, CHUNKS, SMAX>, dim3(n_rows), dim3(threads), 0, stream, a)
    constexpr int SMAX = HB_STREAMS > 0 ? HB_STREAMS : 16;
    if (by_four) {
        constexpr int ONE = HB_STREAMS > 0 ? 1 : 8, TWO = HB_STREAMS > 0 ? 2 : 8;  // the kernel for any number of streams comes in one size
        if (chunks <= ONE) HB_HYPER(4, ONE);
        if (chunks <= TWO) HB_HYPER(4, TWO);
        HB_HYPER(4, 8);
    }
    HB_HYPER(1, 8);
#undef HB_HYPER
}
}  // namespace

// Up to 16 streams; rows of a multiple of four entries (16-byte aligned) may have up to 16,384, others up to 4,096.  `single`: src is [tokens, hidden]
// and stands for every stream.  A result in split-K pieces is float whatever `delta_is_bf16` says; bfloat16 results go with bfloat16 rows.
HB_EXPORT int hb_hyper_connect(const float* src, int single, float* dst, int streams, const void* y0, int splits0, const void* y1, int splits1,
                               long long split_stride, int delta_is_bf16, const float* norm0, const float* norm1, float y_eps, float y_scale, const float* mix,
                               const float* share, const float* read, const float* weight, float eps, void* out, int out_is_bf16, const int* rows, int n_rows,
                               int hidden, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (!src || !weight || !out || (mix && (!y0 || !share)) || splits0 < 0 || splits1 < 0 || (rows && dst)) return HB_BAD_ARGUMENT;
    if (streams < 1 || streams > 16 || (HB_STREAMS > 0 && streams != HB_STREAMS) || hidden <= 0 || hidden > 512 * 32 || (delta_is_bf16 && !out_is_bf16)) return HB_UNSUPPORTED_SIZE;
    if (!mix && dst) return HB_BAD_ARGUMENT;  // nothing is pending: there is nothing new to write
    const uintptr_t all = (uintptr_t)src | (uintptr_t)dst | (uintptr_t)y0 | (uintptr_t)y1 | (uintptr_t)norm0 | (uintptr_t)norm1 | (uintptr_t)weight | (uintptr_t)out;
    const bool by_four = hidden % 4 == 0 && (all & 15) == 0 && (split_stride & 3) == 0;
    const HyperArgs a{src, single, dst, streams, {y0, y1}, {splits0, splits1}, (size_t)split_stride, {norm0, norm1}, y_eps, y_scale, mix, share, read, weight, eps, out, rows, hidden};
    const int pieces = by_four ? hidden / 4 : hidden;
    // the block's size and a thread's share follow from the width alone
    const int threads = pieces <= 128 ? 128 : (pieces <= 256 ? 256 : 512), chunks = (pieces + threads - 1) / threads;
    if (chunks > 8) return HB_UNSUPPORTED_SIZE;
    if (delta_is_bf16) return launch_streams<__nv_bfloat16, __nv_bfloat16>(a, n_rows, by_four, threads, chunks, stream);
    if (out_is_bf16) return launch_streams<float, __nv_bfloat16>(a, n_rows, by_four, threads, chunks, stream);
    return launch_streams<float, float>(a, n_rows, by_four, threads, chunks, stream);
}
