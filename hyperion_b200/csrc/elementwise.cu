// Row-wise kernels of the decoder: embedding lookup, residual add fused with RMSNorm, SwiGLU,
// rotate-half position encoding, and the write of new keys and values into cache pages.
// Each is instantiated for float (the 32-bit path) and for bfloat16 storage; arithmetic is float in
// both. What they compute corresponds to the reference's embedding_gather_bf16, add_rmsnorm_bf16,
// swiglu_rows_bf16, rope_bf16 and kv_append_rows_paged_bf16
// (helios/crates/helios-hal/kernels/elementwise.cu:13,29,42,844; kernels/rmsnorm.cu:66), except
// that the residual stream stays in float and a value is rounded once, when it is stored.
#include "common.cuh"

// ---------------------------------------------------------------- embedding
template <typename TW>
__global__ void embedding_kernel(const TW* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out,
                                 int hidden, int vocab, float scale, int* status) {
    const int t = blockIdx.x;
    const int id = ids[t];
    if (id < 0 || id >= vocab) {
        if (threadIdx.x == 0) atomicOr(status, HB_STATUS_BAD_TOKEN);
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[(size_t)t * hidden + i] = 0.f;
        return;
    }
    const TW* row = table + (size_t)id * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[(size_t)t * hidden + i] = to_float(row[i]) * scale;
}

// bfloat16 rows whose width is a multiple of 8: one 16-byte load and two 16-byte stores per thread.
__global__ void embedding_bf16x8_kernel(const __nv_bfloat16* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out,
                                        int hidden, int vocab, float scale, int* status) {
    const int t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0) atomicOr(status, HB_STATUS_BAD_TOKEN);
    const __nv_bfloat16* row = table + (size_t)(ok ? id : 0) * hidden;
    for (int i = threadIdx.x * 8; i < hidden; i += blockDim.x * 8) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
        if (ok) {
            const uint4 v = *reinterpret_cast<const uint4*>(row + i);
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
            const float2 f0 = __bfloat1622float2(h[0]), f1 = __bfloat1622float2(h[1]), f2 = __bfloat1622float2(h[2]), f3 = __bfloat1622float2(h[3]);
            a = make_float4(f0.x * scale, f0.y * scale, f1.x * scale, f1.y * scale);
            b = make_float4(f2.x * scale, f2.y * scale, f3.x * scale, f3.y * scale);
        }
        *reinterpret_cast<float4*>(out + (size_t)t * hidden + i) = a;
        *reinterpret_cast<float4*>(out + (size_t)t * hidden + i + 4) = b;
    }
}

// out[t] = table[ids[t]] * scale, in float (scale 1 leaves the table's values as they are).
HB_EXPORT int hb_embedding(const void* table, int table_is_bf16, const int* ids, float* out, int tokens, int hidden,
                           int vocab, float scale, int* status, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (table_is_bf16 && hidden % 8 == 0 && (((uintptr_t)table | (uintptr_t)out) & 15) == 0) {
        const int threads = min(512, ((hidden / 8 + 31) / 32) * 32);
        embedding_bf16x8_kernel<<<tokens, threads, 0, stream>>>((const __nv_bfloat16*)table, ids, out, hidden, vocab, scale, status);
        return launch_status();
    }
    if (table_is_bf16)
        embedding_kernel<<<tokens, 256, 0, stream>>>((const __nv_bfloat16*)table, ids, out, hidden, vocab, scale, status);
    else
        embedding_kernel<<<tokens, 256, 0, stream>>>((const float*)table, ids, out, hidden, vocab, scale, status);
    return launch_status();
}

// Tokens that were sampled by the step before and never left the device: ids[pairs[2i]] = source[pairs[2i+1]].
__global__ void place_tokens_kernel(int* __restrict__ ids, const int* __restrict__ source, const int* __restrict__ pairs, int n) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) ids[pairs[2 * i]] = source[pairs[2 * i + 1]];
}

// The caller has checked the pairs against the sizes of ids and source.
HB_EXPORT int hb_place_tokens(int* ids, const int* source, const int* pairs, int n, cudaStream_t stream) {
    if (n <= 0) return 0;
    place_tokens_kernel<<<(n + 127) / 128, 128, 0, stream>>>(ids, source, pairs, n);
    return launch_status();
}

// ---------------------------------------------------------------- residual add + RMSNorm
// Output row r normalises source row s = rows ? rows[r] : r of h (+ delta). With `write_h` the sum
// is stored back into h[s] (the residual stream); it is skipped when rows are gathered for the
// final norm, whose sum nobody reads again. The sum of squares is taken in a fixed order.
template <typename TD, typename TO>
__global__ void add_rmsnorm_kernel(float* __restrict__ h, const TD* __restrict__ delta, const float* __restrict__ weight,
                                   TO* __restrict__ out, const int* __restrict__ rows, int hidden, float eps, int write_h) {
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int s = rows ? rows[r] : r;
    float* hrow = h + (size_t)s * hidden;
    const TD* drow = delta ? delta + (size_t)s * hidden : nullptr;
    float sum = 0.f;
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = hrow[i];
        if (drow) {
            v += to_float(drow[i]);
            if (write_h) hrow[i] = v;
        }
        sum = fmaf(v, v, sum);
    }
    const float total = block_sum(sum, scratch);
    const float inv = 1.0f / sqrtf(total / (float)hidden + eps);
    TO* orow = out + (size_t)r * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = hrow[i];
        if (drow && !write_h) v += to_float(drow[i]);
        orow[i] = from_float<TO>(v * inv * weight[i]);
    }
}

// The same with a row's values held in registers between the two passes (rows of up to 8 values per thread): one trip
// to memory instead of two, which is what counts when a decode step has only a handful of rows.
template <typename TD, typename TO>
__global__ void add_rmsnorm_cached_kernel(float* __restrict__ h, const TD* __restrict__ delta, const float* __restrict__ weight,
                                          TO* __restrict__ out, const int* __restrict__ rows, int hidden, float eps, int write_h) {
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int s = rows ? rows[r] : r;
    float* hrow = h + (size_t)s * hidden;
    const TD* drow = delta ? delta + (size_t)s * hidden : nullptr;
    float v[8], w[8];
    float sum = 0.f;
    let_next_kernel_start();
#pragma unroll
    for (int j = 0; j < 8; ++j) {  // the norm's weight is nobody's output: it is fetched while the kernel before still runs
        const int i = threadIdx.x + j * blockDim.x;
        w[j] = i < hidden ? weight[i] : 0.f;
    }
    wait_for_previous_kernels();
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        v[j] = 0.f;
        if (i < hidden) {
            v[j] = hrow[i];
            if (drow) v[j] += to_float(drow[i]);
        }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {  // the same order of additions per thread as the uncached kernel
        const int i = threadIdx.x + j * blockDim.x;
        if (i < hidden) {
            if (drow && write_h) hrow[i] = v[j];
            sum = fmaf(v[j], v[j], sum);
        }
    }
    const float total = block_sum(sum, scratch);
    const float inv = 1.0f / sqrtf(total / (float)hidden + eps);
    TO* orow = out + (size_t)r * hidden;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i < hidden) orow[i] = from_float<TO>(v[j] * inv * w[j]);
    }
}

// The serving path's shape of it (bfloat16 delta and output, rows of a multiple of 8 values): 8 values per thread and
// group with 16- and 32-byte accesses, each row read once. G groups per thread cover rows of up to 8 * G * 512 values.
// With `partials` ([splits, tokens, hidden] floats: the split-K sums of the product that made the delta) the delta is
// their sum in split order plus the bias, rounded to bfloat16 as the product's own reduction would store it.
// split-K pieces a thread asks for at once (products of a decode step are split 5 to 10 times); fewer where a thread holds
// several groups of a wide row
__host__ __device__ constexpr int pieces_ahead(int groups_per_thread) { return groups_per_thread == 1 ? 12 : (groups_per_thread == 2 ? 8 : 4); }
struct SplitDelta {
    const float* partials;
    size_t split_stride;  // tokens * hidden
    int splits;
    const float* bias_f;
    const __nv_bfloat16* bias_h;
};

template <int G>
__global__ void __launch_bounds__(512) add_rmsnorm_bf16x8_kernel(float* __restrict__ h, const __nv_bfloat16* __restrict__ delta, const SplitDelta split,
                                          const float* __restrict__ weight, __nv_bfloat16* __restrict__ out, const int* __restrict__ rows,
                                          int hidden, float eps, int write_h) {
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int s = rows ? rows[r] : r;
    float* hrow = h + (size_t)s * hidden;
    const __nv_bfloat16* drow = delta + (size_t)s * hidden;
    float v[G][8], w[G][8];
    let_next_kernel_start();
#pragma unroll
    for (int g = 0; g < G; ++g) {  // the norm's weight is nobody's output: it is fetched while the kernel before still runs
        const int i = (threadIdx.x + g * blockDim.x) * 8;
        if (i < hidden) {
            const float4 a = *reinterpret_cast<const float4*>(weight + i), b = *reinterpret_cast<const float4*>(weight + i + 4);
            w[g][0] = a.x; w[g][1] = a.y; w[g][2] = a.z; w[g][3] = a.w; w[g][4] = b.x; w[g][5] = b.y; w[g][6] = b.z; w[g][7] = b.w;
        }
    }
    wait_for_previous_kernels();
    float sum = 0.f;
#pragma unroll
    for (int g = 0; g < G; ++g) {
        const int i = (threadIdx.x + g * blockDim.x) * 8;
        if (i < hidden) {
            const float4 a = *reinterpret_cast<const float4*>(hrow + i), b = *reinterpret_cast<const float4*>(hrow + i + 4);
            uint4 d4;
            if (split.partials) {
                float d[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                const float* first = split.partials + (size_t)s * hidden + i;
                // Every piece is asked for before the first is added: a thread that loads four pieces, adds them and only
                // then loads the next four waits for memory once per group, and a step of a handful of rows is nothing but
                // such waits. The order of the additions stays the order of the splits.
                constexpr int PIECES_AHEAD = pieces_ahead(G);
                float4 p0[PIECES_AHEAD], p1[PIECES_AHEAD];
#pragma unroll
                for (int k = 0; k < PIECES_AHEAD; ++k) {
                    if (k < split.splits) {
                        p0[k] = *reinterpret_cast<const float4*>(first + k * split.split_stride);
                        p1[k] = *reinterpret_cast<const float4*>(first + k * split.split_stride + 4);
                    }
                }
#pragma unroll
                for (int k = 0; k < PIECES_AHEAD; ++k) {
                    if (k < split.splits) {
                        d[0] += p0[k].x; d[1] += p0[k].y; d[2] += p0[k].z; d[3] += p0[k].w;
                        d[4] += p1[k].x; d[5] += p1[k].y; d[6] += p1[k].z; d[7] += p1[k].w;
                    }
                }
                for (int k = PIECES_AHEAD; k < split.splits; ++k) {
                    const float4 q0 = *reinterpret_cast<const float4*>(first + k * split.split_stride);
                    const float4 q1 = *reinterpret_cast<const float4*>(first + k * split.split_stride + 4);
                    d[0] += q0.x; d[1] += q0.y; d[2] += q0.z; d[3] += q0.w; d[4] += q1.x; d[5] += q1.y; d[6] += q1.z; d[7] += q1.w;
                }
                __nv_bfloat162* packed = reinterpret_cast<__nv_bfloat162*>(&d4);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float b0 = split.bias_f ? split.bias_f[i + 2 * e] : (split.bias_h ? __bfloat162float(split.bias_h[i + 2 * e]) : 0.f);
                    const float b1 = split.bias_f ? split.bias_f[i + 2 * e + 1] : (split.bias_h ? __bfloat162float(split.bias_h[i + 2 * e + 1]) : 0.f);
                    packed[e] = __floats2bfloat162_rn(d[2 * e] + b0, d[2 * e + 1] + b1);
                }
            } else {
                d4 = *reinterpret_cast<const uint4*>(drow + i);
            }
            const __nv_bfloat162* d2 = reinterpret_cast<const __nv_bfloat162*>(&d4);
            const float2 d0 = __bfloat1622float2(d2[0]), d1 = __bfloat1622float2(d2[1]), d2f = __bfloat1622float2(d2[2]), d3 = __bfloat1622float2(d2[3]);
            v[g][0] = a.x + d0.x; v[g][1] = a.y + d0.y; v[g][2] = a.z + d1.x; v[g][3] = a.w + d1.y;
            v[g][4] = b.x + d2f.x; v[g][5] = b.y + d2f.y; v[g][6] = b.z + d3.x; v[g][7] = b.w + d3.y;
            if (write_h) {
                *reinterpret_cast<float4*>(hrow + i) = make_float4(v[g][0], v[g][1], v[g][2], v[g][3]);
                *reinterpret_cast<float4*>(hrow + i + 4) = make_float4(v[g][4], v[g][5], v[g][6], v[g][7]);
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) sum = fmaf(v[g][e], v[g][e], sum);
        }
    }
    const float total = block_sum(sum, scratch);
    const float inv = 1.0f / sqrtf(total / (float)hidden + eps);
    __nv_bfloat16* orow = out + (size_t)r * hidden;
#pragma unroll
    for (int g = 0; g < G; ++g) {
        const int i = (threadIdx.x + g * blockDim.x) * 8;
        if (i < hidden) {
            uint4 o4;
            __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o4);
#pragma unroll
            for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(v[g][2 * e] * inv * w[g][2 * e], v[g][2 * e + 1] * inv * w[g][2 * e + 1]);
            *reinterpret_cast<uint4*>(orow + i) = o4;
        }
    }
}

static bool bf16x8_norm_takes(const void* h, const void* delta, const void* weight, const void* out, int hidden) {
    return hidden % 8 == 0 && hidden <= 16384 && (((uintptr_t)h | (uintptr_t)delta | (uintptr_t)weight | (uintptr_t)out) & 15) == 0;
}

static int launch_bf16x8_norm(float* h, const __nv_bfloat16* delta, const SplitDelta& split, const float* weight, __nv_bfloat16* out, const int* rows,
                              int n_rows, int hidden, float eps, int write_h, cudaStream_t stream) {
    const int groups = hidden / 8;
    const int per_thread = groups > 1024 ? 4 : (groups > 512 ? 2 : 1);  // blocks of at most 512 threads: the kernel holds a row's pieces in registers
    const int width = ((groups + per_thread - 1) / per_thread + 31) / 32 * 32;
    if (per_thread == 1)
        return launch_after_previous(add_rmsnorm_bf16x8_kernel<1>, n_rows, width, 0, stream, h, delta, split, weight, out, rows, hidden, eps, write_h);
    if (per_thread == 2)
        return launch_after_previous(add_rmsnorm_bf16x8_kernel<2>, n_rows, width, 0, stream, h, delta, split, weight, out, rows, hidden, eps, write_h);
    return launch_after_previous(add_rmsnorm_bf16x8_kernel<4>, n_rows, width, 0, stream, h, delta, split, weight, out, rows, hidden, eps, write_h);
}

// The same with the delta still in pieces: partials [splits, tokens, hidden] floats (+ a bias) are added up in split order
// and rounded to bfloat16 before they join the residual stream. Refuses (HB_UNSUPPORTED_SIZE) what the 8-wide kernel cannot take.
HB_EXPORT int hb_add_rmsnorm_splits(float* h, const float* partials, int splits, int tokens, const float* bias_f, const void* bias_h,
                                    const float* weight, void* out, const int* rows, int n_rows, int hidden, float eps, int write_h,
                                    cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (!partials || splits < 1 || tokens < 1) return HB_BAD_ARGUMENT;
    if (!bf16x8_norm_takes(h, partials, weight, out, hidden)) return HB_UNSUPPORTED_SIZE;
    const SplitDelta split{partials, (size_t)tokens * hidden, splits, bias_f, (const __nv_bfloat16*)bias_h};
    return launch_bf16x8_norm(h, nullptr, split, weight, (__nv_bfloat16*)out, rows, n_rows, hidden, eps, write_h, stream);
}

HB_EXPORT int hb_add_rmsnorm(float* h, const void* delta, int delta_is_bf16, const float* weight, void* out,
                             int out_is_bf16, const int* rows, int n_rows, int hidden, float eps, int write_h,
                             cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (delta && delta_is_bf16 && out_is_bf16 && bf16x8_norm_takes(h, delta, weight, out, hidden))
        return launch_bf16x8_norm(h, (const __nv_bfloat16*)delta, SplitDelta{nullptr, 0, 0, nullptr, nullptr}, weight, (__nv_bfloat16*)out, rows, n_rows,
                                  hidden, eps, write_h, stream);
    const int threads = hidden >= 4096 ? 1024 : (hidden >= 1024 ? 512 : 256);
    int status = 0;
    const bool cached = hidden <= 8 * threads;  // both kernels add a thread's squares in the same order, so they agree bit for bit
#define HB_NORM(TD, TO)                                                                                                                    \
    if (cached) status = launch_after_previous(add_rmsnorm_cached_kernel<TD, TO>, n_rows, threads, 0, stream, h, (const TD*)delta, weight, (TO*)out, rows, hidden, eps, write_h); \
    else status = launch_after_previous(add_rmsnorm_kernel<TD, TO>, n_rows, threads, 0, stream, h, (const TD*)delta, weight, (TO*)out, rows, hidden, eps, write_h)
    if (delta_is_bf16) {
        if (out_is_bf16) { HB_NORM(__nv_bfloat16, __nv_bfloat16); } else { HB_NORM(__nv_bfloat16, float); }
    } else {
        if (out_is_bf16) { HB_NORM(float, __nv_bfloat16); } else { HB_NORM(float, float); }
    }
#undef HB_NORM
    return status;
}

// ---------------------------------------------------------------- SwiGLU
// in: [tokens, 2*inter]: gate and up columns alternate in blocks of `block` columns (block gate columns, then the block up
// columns that belong to them; block = inter is the plain arrangement, all gate columns first);
// out[t, i] = silu(gate_i) * up_i, silu(g) = g / (1 + exp(-g)) in float.
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int inter, int block) {
    const int t = blockIdx.y;
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= inter) return;
    const size_t at = (size_t)t * 2 * inter + (size_t)(i / block) * 2 * block + i % block;
    const float g = to_float(gate_up[at]);
    const float u = to_float(gate_up[at + block]);
    out[(size_t)t * inter + i] = from_float<T>(g / (1.0f + expf(-g)) * u);
}

// bfloat16 rows whose width and block are multiples of 8: 16-byte loads and stores, 8 elements per thread.
__global__ void swiglu_bf16x8_kernel(const __nv_bfloat16* __restrict__ gate_up, __nv_bfloat16* __restrict__ out, int inter, int block) {
    const int t = blockIdx.y;
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    let_next_kernel_start();
    wait_for_previous_kernels();
    if (i >= inter) return;
    const size_t at = (size_t)t * 2 * inter + (size_t)(i / block) * 2 * block + i % block;
    const uint4 g4 = *reinterpret_cast<const uint4*>(gate_up + at);
    const uint4 u4 = *reinterpret_cast<const uint4*>(gate_up + at + block);
    const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&g4);
    const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&u4);
    uint4 o4;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o4);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 g = __bfloat1622float2(g2[e]), u = __bfloat1622float2(u2[e]);
        o2[e] = __floats2bfloat162_rn(g.x / (1.0f + expf(-g.x)) * u.x, g.y / (1.0f + expf(-g.y)) * u.y);
    }
    *reinterpret_cast<uint4*>(out + (size_t)t * inter + i) = o4;
}

// block: columns per run of gate (and of up) columns; it divides inter (inter itself: all gate columns first).
HB_EXPORT int hb_swiglu(const void* gate_up, void* out, int is_bf16, int tokens, int inter, int block, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (tokens > 65535) return HB_UNSUPPORTED_SIZE;
    if (block <= 0 || inter % block) return HB_BAD_ARGUMENT;
    if (is_bf16 && inter % 8 == 0 && block % 8 == 0 && (((uintptr_t)gate_up | (uintptr_t)out) & 15) == 0) {
        dim3 grid8((inter / 8 + 255) / 256, tokens);
        return launch_after_previous(swiglu_bf16x8_kernel, grid8, 256, 0, stream, (const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, inter, block);
    }
    dim3 grid((inter + 255) / 256, tokens);
    if (is_bf16)
        swiglu_kernel<<<grid, 256, 0, stream>>>((const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, inter, block);
    else
        swiglu_kernel<<<grid, 256, 0, stream>>>((const float*)gate_up, (float*)out, inter, block);
    return launch_status();
}

// ---------------------------------------------------------------- rotate-half position encoding
// Rotates `heads` consecutive heads of `head_dim` columns at the start of every row of `x` (row
// stride `stride` elements), in place: y[i] = x[i] c - x[i+d/2] s, y[i+d/2] = x[i+d/2] c + x[i] s
// with (c, s) = table[position][i]. The table holds cos and sin of position * base^(-2i/d).
template <typename T>
__global__ void rope_kernel(T* __restrict__ x, const int* __restrict__ positions, const float2* __restrict__ table,
                            int stride, int heads, int head_dim, int max_positions, int* status) {
    const int t = blockIdx.x;
    const int half = head_dim >> 1;
    const int pos = positions[t];
    if (pos < 0 || pos >= max_positions) {
        if (threadIdx.x == 0) atomicOr(status, HB_STATUS_BAD_POSITION);
        return;
    }
    T* row = x + (size_t)t * stride;
    const float2* cs = table + (size_t)pos * half;
    for (int e = threadIdx.x; e < heads * half; e += blockDim.x) {
        const int head = e / half, i = e - head * half;
        const float2 c = cs[i];
        T* p = row + head * head_dim + i;
        const float x1 = to_float(p[0]), x2 = to_float(p[half]);
        p[0] = from_float<T>(x1 * c.x - x2 * c.y);
        p[half] = from_float<T>(x2 * c.x + x1 * c.y);
    }
}

HB_EXPORT int hb_rope(void* x, int is_bf16, const int* positions, const float* table, int tokens, int stride, int heads,
                      int head_dim, int max_positions, int* status, cudaStream_t stream) {
    if (tokens <= 0 || heads <= 0) return 0;
    if (head_dim & 1) return HB_UNSUPPORTED_SIZE;
    if (is_bf16)
        rope_kernel<<<tokens, 256, 0, stream>>>((__nv_bfloat16*)x, positions, (const float2*)table, stride, heads, head_dim, max_positions, status);
    else
        rope_kernel<<<tokens, 256, 0, stream>>>((float*)x, positions, (const float2*)table, stride, heads, head_dim, max_positions, status);
    return launch_status();
}

// ---------------------------------------------------------------- key/value write into pages
// One cache layer is [pages, 2, kv_heads, page_size, head_dim]. Token t of row r = token_row[t] at
// position p goes to page block_table[r][p / page_size], slot p % page_size. A missing page sets
// the status word and the token is skipped.
template <typename T>
__global__ void kv_store_kernel(const T* __restrict__ src, int stride, int k_offset, int v_offset, T* __restrict__ cache,
                                const int* __restrict__ block_table, int table_width, const int* __restrict__ token_row,
                                const int* __restrict__ positions, int kv_heads, int head_dim, int page_size, int pages,
                                int* status) {
    const int t = blockIdx.x;
    const int pos = positions[t];
    const int block = pos / page_size;
    const int page = (block < table_width && pos >= 0) ? block_table[(size_t)token_row[t] * table_width + block] : -1;
    if (page < 0 || page >= pages) {
        if (threadIdx.x == 0) atomicOr(status, HB_STATUS_BAD_PAGE);
        return;
    }
    const int slot = pos - block * page_size;
    const int width = kv_heads * head_dim;
    const T* row = src + (size_t)t * stride;
    const size_t page_base = (size_t)page * 2 * kv_heads * page_size * head_dim;
    for (int e = threadIdx.x; e < 2 * width; e += blockDim.x) {
        const int which = e / width, c = e - which * width;
        const int head = c / head_dim, d = c - head * head_dim;
        const T v = row[(which ? v_offset : k_offset) + c];
        cache[page_base + (((size_t)which * kv_heads + head) * page_size + slot) * head_dim + d] = v;
    }
}

// ---------------------------------------------------------------- rotation fused with the cache write
// One pass over a token's [q | k | v] row: the query heads are rotated in place, the key heads are
// rotated on their way into the cache (the row's own copy of k is left as it was: nothing reads it
// again), the value heads are copied.  Same arithmetic as rope_kernel followed by kv_store_kernel.
template <typename T>
__global__ void rope_kv_store_kernel(T* __restrict__ x, int stride, int q_heads, int kv_heads, int head_dim,
                                     const int* __restrict__ positions, const float2* __restrict__ table, int max_positions,
                                     T* __restrict__ cache, const int* __restrict__ block_table, int table_width,
                                     const int* __restrict__ token_row, int page_size, int pages, int* status) {
    const int t = blockIdx.x;
    const int half = head_dim >> 1;
    const int pos = positions[t];
    if (pos < 0 || pos >= max_positions) {
        if (threadIdx.x == 0) atomicOr(status, HB_STATUS_BAD_POSITION);
        return;
    }
    const int block = pos / page_size;
    const int page = block < table_width ? block_table[(size_t)token_row[t] * table_width + block] : -1;
    const bool page_ok = page >= 0 && page < pages;
    if (!page_ok && threadIdx.x == 0 && blockIdx.y == 0) atomicOr(status, HB_STATUS_BAD_PAGE);
    const int slot = pos - block * page_size;
    T* row = x + (size_t)t * stride;
    const float2* cs = table + (size_t)pos * half;
    const size_t page_base = (size_t)(page_ok ? page : 0) * 2 * kv_heads * page_size * head_dim;
    const int rotated = (q_heads + kv_heads) * half;
    // blockIdx.y cuts a token's work into slices of blockDim.x element pairs, so that a decode step of a few tokens
    // still spreads over many blocks
    for (int e = blockIdx.y * blockDim.x + threadIdx.x; e < rotated + kv_heads * half; e += gridDim.y * blockDim.x) {
        if (e < rotated) {
            const int head = e / half, i = e - head * half;
            const float2 c = cs[i];
            T* p = row + head * head_dim + i;
            const float x1 = to_float(p[0]), x2 = to_float(p[half]);
            const T y1 = from_float<T>(x1 * c.x - x2 * c.y), y2 = from_float<T>(x2 * c.x + x1 * c.y);
            if (head < q_heads) {
                p[0] = y1; p[half] = y2;
            } else if (page_ok) {
                T* dst = cache + page_base + (((size_t)(head - q_heads)) * page_size + slot) * head_dim + i;
                dst[0] = y1; dst[half] = y2;
            }
        } else if (page_ok) {  // values: two elements per thread
            const int f = e - rotated, head = f / half, i = (f - head * half) * 2;
            const T* p = row + (q_heads + kv_heads + head) * head_dim + i;
            T* dst = cache + page_base + (((size_t)(kv_heads + head)) * page_size + slot) * head_dim + i;
            dst[0] = p[0]; dst[1] = p[1];
        }
    }
}

// bfloat16 with head sizes that are multiples of 16: every thread rotates 8 consecutive pairs (two 16-byte loads, two
// 16-byte stores) or copies 8 values; same arithmetic per element as the scalar kernel.
__global__ void rope_kv_store_bf16x8_kernel(__nv_bfloat16* __restrict__ x, int stride, int q_heads, int kv_heads, int head_dim,
                                            const int* __restrict__ positions, const float2* __restrict__ table, int max_positions,
                                            __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_table, int table_width,
                                            const int* __restrict__ token_row, int page_size, int pages, int* status) {
    const int t = blockIdx.x;
    const int half = head_dim >> 1, chunks = half >> 3;  // 8-pair chunks per head
    let_next_kernel_start();
    const int pos = positions[t];  // positions and tables come with the step's one copy from the host, not from a kernel
    const bool pos_ok = pos >= 0 && pos < max_positions;
    const int block = pos_ok ? pos / page_size : 0;
    const int page = pos_ok && block < table_width ? block_table[(size_t)token_row[t] * table_width + block] : -1;
    wait_for_previous_kernels();
    if (!pos_ok) {
        if (threadIdx.x == 0 && blockIdx.y == 0) atomicOr(status, HB_STATUS_BAD_POSITION);
        return;
    }
    const bool page_ok = page >= 0 && page < pages;
    if (!page_ok && threadIdx.x == 0 && blockIdx.y == 0) atomicOr(status, HB_STATUS_BAD_PAGE);
    const int slot = pos - block * page_size;
    __nv_bfloat16* row = x + (size_t)t * stride;
    const float2* cs = table + (size_t)pos * half;
    const size_t page_base = (size_t)(page_ok ? page : 0) * 2 * kv_heads * page_size * head_dim;
    const int rotated = (q_heads + kv_heads) * chunks;
    const int total = rotated + kv_heads * 2 * chunks;  // values: head_dim / 8 chunks per head
    for (int e = blockIdx.y * blockDim.x + threadIdx.x; e < total; e += gridDim.y * blockDim.x) {
        if (e < rotated) {
            const int head = e / chunks, i = (e - head * chunks) * 8;
            __nv_bfloat16* p = row + head * head_dim + i;
            const uint4 lo4 = *reinterpret_cast<const uint4*>(p), hi4 = *reinterpret_cast<const uint4*>(p + half);
            const __nv_bfloat16* lo = reinterpret_cast<const __nv_bfloat16*>(&lo4);
            const __nv_bfloat16* hi = reinterpret_cast<const __nv_bfloat16*>(&hi4);
            uint4 out_lo, out_hi;
            __nv_bfloat16* y1 = reinterpret_cast<__nv_bfloat16*>(&out_lo);
            __nv_bfloat16* y2 = reinterpret_cast<__nv_bfloat16*>(&out_hi);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float2 c = cs[i + j];
                const float x1 = __bfloat162float(lo[j]), x2 = __bfloat162float(hi[j]);
                y1[j] = __float2bfloat16_rn(x1 * c.x - x2 * c.y);
                y2[j] = __float2bfloat16_rn(x2 * c.x + x1 * c.y);
            }
            if (head < q_heads) {
                *reinterpret_cast<uint4*>(p) = out_lo;
                *reinterpret_cast<uint4*>(p + half) = out_hi;
            } else if (page_ok) {
                __nv_bfloat16* dst = cache + page_base + (((size_t)(head - q_heads)) * page_size + slot) * head_dim + i;
                *reinterpret_cast<uint4*>(dst) = out_lo;
                *reinterpret_cast<uint4*>(dst + half) = out_hi;
            }
        } else if (page_ok) {
            const int f = e - rotated, head = f / (2 * chunks), i = (f - head * 2 * chunks) * 8;
            const uint4 v = *reinterpret_cast<const uint4*>(row + (q_heads + kv_heads + head) * head_dim + i);
            *reinterpret_cast<uint4*>(cache + page_base + (((size_t)(kv_heads + head)) * page_size + slot) * head_dim + i) = v;
        }
    }
}

HB_EXPORT int hb_rope_kv_store(void* x, int is_bf16, int tokens, int stride, int q_heads, int kv_heads, int head_dim,
                               const int* positions, const float* table, int max_positions, void* cache, const int* block_table,
                               int table_width, const int* token_row, int page_size, int pages, int* status, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (head_dim & 1) return HB_UNSUPPORTED_SIZE;
    if (is_bf16 && head_dim % 16 == 0 && stride % 8 == 0 && (((uintptr_t)x | (uintptr_t)cache) & 15) == 0) {
        const int items = (q_heads + 2 * kv_heads) * (head_dim / 16);
        const int threads = items >= 256 ? 256 : 128;
        const dim3 grid8(tokens, tokens >= 512 ? 1 : min(8, (items + threads - 1) / threads));
        return launch_after_previous(rope_kv_store_bf16x8_kernel, grid8, threads, 0, stream, (__nv_bfloat16*)x, stride, q_heads, kv_heads, head_dim,
                                     positions, (const float2*)table, max_positions, (__nv_bfloat16*)cache, block_table, table_width, token_row,
                                     page_size, pages, status);
    }
    const int pairs = (q_heads + 2 * kv_heads) * (head_dim / 2);
    const int slices = tokens >= 512 ? 1 : min(16, (pairs + 255) / 256);
    const dim3 grid(tokens, slices);
    if (is_bf16)
        rope_kv_store_kernel<<<grid, 256, 0, stream>>>((__nv_bfloat16*)x, stride, q_heads, kv_heads, head_dim, positions, (const float2*)table,
                                                       max_positions, (__nv_bfloat16*)cache, block_table, table_width, token_row, page_size, pages, status);
    else
        rope_kv_store_kernel<<<grid, 256, 0, stream>>>((float*)x, stride, q_heads, kv_heads, head_dim, positions, (const float2*)table,
                                                       max_positions, (float*)cache, block_table, table_width, token_row, page_size, pages, status);
    return launch_status();
}

HB_EXPORT int hb_kv_store(const void* src, int is_bf16, int tokens, int stride, int k_offset, int v_offset, void* cache,
                          const int* block_table, int table_width, const int* token_row, const int* positions,
                          int kv_heads, int head_dim, int page_size, int pages, int* status, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (is_bf16)
        kv_store_kernel<<<tokens, 256, 0, stream>>>((const __nv_bfloat16*)src, stride, k_offset, v_offset, (__nv_bfloat16*)cache,
                                                    block_table, table_width, token_row, positions, kv_heads, head_dim, page_size, pages, status);
    else
        kv_store_kernel<<<tokens, 256, 0, stream>>>((const float*)src, stride, k_offset, v_offset, (float*)cache, block_table,
                                                    table_width, token_row, positions, kv_heads, head_dim, page_size, pages, status);
    return launch_status();
}

// ---------------------------------------------------------------- RMSNorm of a sublayer's output, added to the stream
// h[t] += y[t] / sqrt(mean(y[t]^2) + eps) * weight, for blocks that normalise what a sublayer returns instead of what it
// reads.  `copy` (optional) receives the new h[t] in the activation type: the next sublayer's input.  The sum of squares is
// taken in a fixed order per row, so a row's result depends on nothing else in the launch.
template <typename TY, typename TC>
__global__ void rmsnorm_add_kernel(float* __restrict__ h, const TY* __restrict__ y, const float* __restrict__ weight,
                                   TC* __restrict__ copy, int hidden, float eps) {
    __shared__ float scratch[32];
    const int t = blockIdx.x;
    float* hrow = h + (size_t)t * hidden;
    const TY* yrow = y + (size_t)t * hidden;
    float sum = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = to_float(yrow[i]);
        sum = fmaf(v, v, sum);
    }
    const float total = block_sum(sum, scratch);
    const float inv = 1.0f / sqrtf(total / (float)hidden + eps);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = hrow[i] + to_float(yrow[i]) * inv * weight[i];
        hrow[i] = v;
        if (copy) copy[(size_t)t * hidden + i] = from_float<TC>(v);
    }
}

// bfloat16 sublayer outputs in rows of up to 8,192 values, a multiple of 8: a thread keeps its 8 values in registers between the
// sum of squares and the add (one trip to memory), with 16-byte accesses.
__global__ void rmsnorm_add_bf16x8_kernel(float* __restrict__ h, const __nv_bfloat16* __restrict__ y, const float* __restrict__ weight,
                                          __nv_bfloat16* __restrict__ copy, int hidden, float eps) {
    __shared__ float scratch[32];
    const int t = blockIdx.x, i = threadIdx.x * 8;
    const bool active = i < hidden;
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (active) {
        const uint4 raw = *reinterpret_cast<const uint4*>(y + (size_t)t * hidden + i);
        const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(pairs[k]);
            v[2 * k] = f.x; v[2 * k + 1] = f.y;
        }
    }
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) sum = fmaf(v[k], v[k], sum);
    const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps);
    if (!active) return;
    float* hrow = h + (size_t)t * hidden + i;
    float4 h0 = *reinterpret_cast<const float4*>(hrow), h1 = *reinterpret_cast<const float4*>(hrow + 4);
    const float4 w0 = *reinterpret_cast<const float4*>(weight + i), w1 = *reinterpret_cast<const float4*>(weight + i + 4);
    h0.x += v[0] * inv * w0.x; h0.y += v[1] * inv * w0.y; h0.z += v[2] * inv * w0.z; h0.w += v[3] * inv * w0.w;
    h1.x += v[4] * inv * w1.x; h1.y += v[5] * inv * w1.y; h1.z += v[6] * inv * w1.z; h1.w += v[7] * inv * w1.w;
    *reinterpret_cast<float4*>(hrow) = h0;
    *reinterpret_cast<float4*>(hrow + 4) = h1;
    if (copy) {
        uint4 packed;
        __nv_bfloat162* out = reinterpret_cast<__nv_bfloat162*>(&packed);
        out[0] = __floats2bfloat162_rn(h0.x, h0.y); out[1] = __floats2bfloat162_rn(h0.z, h0.w);
        out[2] = __floats2bfloat162_rn(h1.x, h1.y); out[3] = __floats2bfloat162_rn(h1.z, h1.w);
        *reinterpret_cast<uint4*>(copy + (size_t)t * hidden + i) = packed;
    }
}

HB_EXPORT int hb_rmsnorm_add(float* h, const void* y, int y_is_bf16, const float* weight, void* copy, int tokens, int hidden,
                             float eps, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (y_is_bf16 && hidden % 8 == 0 && hidden <= 8192 && (((uintptr_t)h | (uintptr_t)y | (uintptr_t)weight | (uintptr_t)copy) & 15) == 0) {
        const int lanes = ((hidden / 8 + 31) / 32) * 32;  // which kernel runs follows from the width alone
        rmsnorm_add_bf16x8_kernel<<<tokens, lanes, 0, stream>>>(h, (const __nv_bfloat16*)y, weight, (__nv_bfloat16*)copy, hidden, eps);
        return launch_status();
    }
    const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
    if (y_is_bf16)
        rmsnorm_add_kernel<<<tokens, threads, 0, stream>>>(h, (const __nv_bfloat16*)y, weight, (__nv_bfloat16*)copy, hidden, eps);
    else
        rmsnorm_add_kernel<<<tokens, threads, 0, stream>>>(h, (const float*)y, weight, (float*)nullptr, hidden, eps);
    return launch_status();
}

// The float stream in the activation type (bfloat16): what the first sublayer of a model reads.
__global__ void stream_copy_kernel(const float* __restrict__ h, __nv_bfloat16* __restrict__ copy, size_t count) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (size_t)gridDim.x * blockDim.x)
        copy[i] = __float2bfloat16_rn(h[i]);
}

HB_EXPORT int hb_stream_copy(const float* h, void* copy, long long count, cudaStream_t stream) {
    if (count <= 0) return 0;
    const int blocks = (int)((count + 255) / 256 < 4096 ? (count + 255) / 256 : 4096);
    stream_copy_kernel<<<blocks, 256, 0, stream>>>(h, (__nv_bfloat16*)copy, (size_t)count);
    return launch_status();
}

// ---------------------------------------------------------------- norm of a sublayer's output + residual add + the next sublayer's norm
// For blocks that normalise both what a sublayer reads and what it returns (x <- x + norm_b(f(norm_a(x)))), one launch per
// sublayer boundary:   h[t] += y[t] / sqrt(mean(y[t]^2) + eps) * w_post (+ offset);   out[i] = h[t] / sqrt(mean(h[t]^2) + eps) * w_next.
// Every piece is optional: without y only the offset is added, without w_next nothing is normalised for a reader.  With `rows`
// only the listed rows are worked on and h is left as it was (the last norm of a model, where only some rows are read).
// With `gate` [tokens, gate_stride] (float) the sublayer's output is first multiplied, entry by entry, by sigmoid(gate[t] + gate_bias): a block whose
// sublayers are gated by a projection of what they read hands the projection on instead of launching the product itself.  The projection may
// still lie in `gate_splits` split-K pieces, `gate_split_stride` floats apart, which are added up here in split order, after the bias.
// Everything is float; sums of squares are taken in a fixed order per row.
template <typename TY, typename TO>
__global__ void norm_add_norm_kernel(float* __restrict__ h, const TY* __restrict__ y, const float* __restrict__ w_post,
                                     const float* __restrict__ offset, const float* __restrict__ w_next, TO* __restrict__ out,
                                     const int* __restrict__ rows, int hidden, float eps_post, float eps_next, const float* __restrict__ gate,
                                     int gate_stride, int gate_splits, size_t gate_split_stride, const float* __restrict__ gate_bias) {
    extern __shared__ float row_values[];
    __shared__ float scratch[32];
    const int i = blockIdx.x, t = rows ? rows[i] : i;
    float* hrow = h + (size_t)t * hidden;
    const TY* yrow = y ? y + (size_t)t * hidden : nullptr;
    const float* grow = (y && gate) ? gate + (size_t)t * gate_stride : nullptr;
    float inv_y = 0.f;
    if (yrow) {
        float sum = 0.f;
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
            float v = to_float(yrow[j]);
            if (grow) {
                float g = gate_bias ? gate_bias[j] : 0.f;
                for (int piece = 0; piece < gate_splits; ++piece) g += grow[(size_t)piece * gate_split_stride + j];
                const float open = 1.0f / (1.0f + expf(-g));
                v *= open;
                row_values[j] = open;  // kept for the second pass over the row
            }
            sum = fmaf(v, v, sum);
        }
        inv_y = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps_post);
    }
    float sum = 0.f;
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
        float v = hrow[j];
        if (yrow) v += to_float(yrow[j]) * (grow ? row_values[j] : 1.f) * inv_y * w_post[j];
        if (offset) v += offset[j];
        row_values[j] = v;
        if (!rows) hrow[j] = v;
        sum = fmaf(v, v, sum);
    }
    if (!w_next) return;
    const float inv_h = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps_next);
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) out[(size_t)i * hidden + j] = from_float<TO>(row_values[j] * inv_h * w_next[j]);
}

// The same for bfloat16 sublayer outputs and readers in rows of up to 8,192 values, a multiple of 8: a thread keeps its 8 values
// in registers through both norms (one trip to memory), with 16-byte accesses.
__global__ void norm_add_norm_bf16x8_kernel(float* __restrict__ h, const __nv_bfloat16* __restrict__ y, const float* __restrict__ w_post,
                                            const float* __restrict__ offset, const float* __restrict__ w_next, __nv_bfloat16* __restrict__ out,
                                            const int* __restrict__ rows, int hidden, float eps_post, float eps_next, const float* __restrict__ gate,
                                            int gate_stride, int gate_splits, size_t gate_split_stride, const float* __restrict__ gate_bias) {
    __shared__ float scratch[32];
    const int i = blockIdx.x, t = rows ? rows[i] : i, j = threadIdx.x * 8;
    const bool active = j < hidden;
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    float inv_y = 0.f;
    if (y) {
        if (active) {
            const uint4 raw = *reinterpret_cast<const uint4*>(y + (size_t)t * hidden + j);
            const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(pairs[k]);
                v[2 * k] = f.x; v[2 * k + 1] = f.y;
            }
            if (gate) {
                float g[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
                if (gate_bias) {
                    const float4 b0 = *reinterpret_cast<const float4*>(gate_bias + j), b1 = *reinterpret_cast<const float4*>(gate_bias + j + 4);
                    g[0] = b0.x; g[1] = b0.y; g[2] = b0.z; g[3] = b0.w; g[4] = b1.x; g[5] = b1.y; g[6] = b1.z; g[7] = b1.w;
                }
                for (int piece = 0; piece < gate_splits; ++piece) {
                    const float* grow = gate + (size_t)piece * gate_split_stride + (size_t)t * gate_stride + j;
                    const float4 g0 = *reinterpret_cast<const float4*>(grow), g1 = *reinterpret_cast<const float4*>(grow + 4);
                    g[0] += g0.x; g[1] += g0.y; g[2] += g0.z; g[3] += g0.w; g[4] += g1.x; g[5] += g1.y; g[6] += g1.z; g[7] += g1.w;
                }
#pragma unroll
                for (int k = 0; k < 8; ++k) v[k] *= 1.0f / (1.0f + expf(-g[k]));
            }
        }
        float sum = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) sum = fmaf(v[k], v[k], sum);
        inv_y = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps_post);
    }
    float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    float* hrow = h + (size_t)t * hidden + j;
    if (active) {
        const float4 h0 = *reinterpret_cast<const float4*>(hrow), h1 = *reinterpret_cast<const float4*>(hrow + 4);
        x[0] = h0.x; x[1] = h0.y; x[2] = h0.z; x[3] = h0.w; x[4] = h1.x; x[5] = h1.y; x[6] = h1.z; x[7] = h1.w;
        if (y) {
            const float4 w0 = *reinterpret_cast<const float4*>(w_post + j), w1 = *reinterpret_cast<const float4*>(w_post + j + 4);
            const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
            for (int k = 0; k < 8; ++k) x[k] += v[k] * inv_y * w[k];
        }
        if (offset) {
            const float4 o0 = *reinterpret_cast<const float4*>(offset + j), o1 = *reinterpret_cast<const float4*>(offset + j + 4);
            x[0] += o0.x; x[1] += o0.y; x[2] += o0.z; x[3] += o0.w; x[4] += o1.x; x[5] += o1.y; x[6] += o1.z; x[7] += o1.w;
        }
        if (!rows) {
            *reinterpret_cast<float4*>(hrow) = make_float4(x[0], x[1], x[2], x[3]);
            *reinterpret_cast<float4*>(hrow + 4) = make_float4(x[4], x[5], x[6], x[7]);
        }
    }
    if (!w_next) return;
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) sum = fmaf(x[k], x[k], sum);
    const float inv_h = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps_next);
    if (!active) return;
    const float4 n0 = *reinterpret_cast<const float4*>(w_next + j), n1 = *reinterpret_cast<const float4*>(w_next + j + 4);
    uint4 packed;
    __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&packed);
    o[0] = __floats2bfloat162_rn(x[0] * inv_h * n0.x, x[1] * inv_h * n0.y);
    o[1] = __floats2bfloat162_rn(x[2] * inv_h * n0.z, x[3] * inv_h * n0.w);
    o[2] = __floats2bfloat162_rn(x[4] * inv_h * n1.x, x[5] * inv_h * n1.y);
    o[3] = __floats2bfloat162_rn(x[6] * inv_h * n1.z, x[7] * inv_h * n1.w);
    *reinterpret_cast<uint4*>(out + (size_t)i * hidden + j) = packed;
}

HB_EXPORT int hb_norm_add_norm(float* h, const void* y, int y_is_bf16, const float* w_post, const float* offset, const float* w_next, void* out,
                               int out_is_bf16, const int* rows, int n_rows, int hidden, float eps_post, float eps_next, const float* gate,
                               int gate_stride, int gate_splits, long long gate_split_stride, const float* gate_bias, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (hidden <= 0 || hidden > 49152 || (y && !w_post) || (w_next && !out) || (gate && gate_splits < 1)) return HB_BAD_ARGUMENT;
    const bool halves = (!y || y_is_bf16) && (!w_next || out_is_bf16);
    if (halves && hidden % 8 == 0 && hidden <= 8192 && (!gate || (gate_stride % 4 == 0 && gate_split_stride % 4 == 0)) &&
        (((uintptr_t)h | (uintptr_t)y | (uintptr_t)w_post | (uintptr_t)offset | (uintptr_t)w_next | (uintptr_t)out | (uintptr_t)gate | (uintptr_t)gate_bias) & 15) == 0) {
        const int lanes = ((hidden / 8 + 31) / 32) * 32;  // which kernel runs follows from the width and the types alone
        norm_add_norm_bf16x8_kernel<<<n_rows, lanes, 0, stream>>>(h, (const __nv_bfloat16*)y, w_post, offset, w_next, (__nv_bfloat16*)out, rows, hidden,
                                                                  eps_post, eps_next, gate, gate_stride, gate_splits, (size_t)gate_split_stride, gate_bias);
        return launch_status();
    }
    const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
    const size_t shared = (size_t)hidden * sizeof(float);
#define HB_NORM_ADD_NORM(TY, TO)                                                                                                          \
    do {                                                                                                                                  \
        if (shared > 48 * 1024) cudaFuncSetAttribute(norm_add_norm_kernel<TY, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared); \
        norm_add_norm_kernel<TY, TO><<<n_rows, threads, shared, stream>>>(h, (const TY*)y, w_post, offset, w_next, (TO*)out, rows, hidden,   \
                                                                         eps_post, eps_next, gate, gate_stride, gate_splits,            \
                                                                         (size_t)gate_split_stride, gate_bias);                          \
    } while (0)
    const bool y16 = y && y_is_bf16, o16 = w_next && out_is_bf16;
    if (y16 && o16) HB_NORM_ADD_NORM(__nv_bfloat16, __nv_bfloat16);
    else if (y16) HB_NORM_ADD_NORM(__nv_bfloat16, float);
    else if (o16) HB_NORM_ADD_NORM(float, __nv_bfloat16);
    else HB_NORM_ADD_NORM(float, float);
#undef HB_NORM_ADD_NORM
    return launch_status();
}

// ---------------------------------------------------------------- GELU in its tanh form
// out = 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), in float, rounded once.
template <typename T>
__global__ void gelu_tanh_kernel(const T* __restrict__ x, T* __restrict__ out, size_t count) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (size_t)gridDim.x * blockDim.x) {
        const float z = to_float(x[i]);
        out[i] = from_float<T>(0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))));
    }
}

HB_EXPORT int hb_gelu_tanh(const void* x, void* out, int is_bf16, long long count, cudaStream_t stream) {
    if (count <= 0) return 0;
    const int blocks = (int)((count + 255) / 256 < 8192 ? (count + 255) / 256 : 8192);
    if (is_bf16) gelu_tanh_kernel<<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)out, (size_t)count);
    else gelu_tanh_kernel<<<blocks, 256, 0, stream>>>((const float*)x, (float*)out, (size_t)count);
    return launch_status();
}

// ---------------------------------------------------------------- a sigmoid gate on rows, in place
// x[t, c] <- x[t, c] * scale * sigmoid(gate[t, gate_off + c]) for c < width; the gate is float, the product is rounded once.
template <typename T>
__global__ void sigmoid_gate_kernel(T* __restrict__ x, int x_stride, const float* __restrict__ gate, int gate_stride, int gate_off, float scale, int width) {
    const int t = blockIdx.y;
    for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < width; c += gridDim.x * blockDim.x) {
        const float g = gate[(size_t)t * gate_stride + gate_off + c];
        x[(size_t)t * x_stride + c] = from_float<T>(to_float(x[(size_t)t * x_stride + c]) * (scale / (1.f + expf(-g))));
    }
}

// Four columns per access, for rows of whole pieces.
template <typename T>
__global__ void sigmoid_gate4_kernel(T* __restrict__ x, int x_stride, const float* __restrict__ gate, int gate_stride, int gate_off, float scale, int width) {
    const int t = blockIdx.y, c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (c >= width) return;
    float g[4], v[4];
    load4(gate + (size_t)t * gate_stride + gate_off + c, g);
    load4(x + (size_t)t * x_stride + c, v);
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] *= scale / (1.f + expf(-g[e]));
    store4(x + (size_t)t * x_stride + c, v);
}

HB_EXPORT int hb_sigmoid_gate(void* x, int is_bf16, int x_stride, const float* gate, int gate_stride, int gate_off, float scale, int tokens, int width,
                              cudaStream_t stream) {
    if (tokens <= 0 || width <= 0) return 0;
    for (int first = 0; first < tokens; first += 65535) {
        const int count = tokens - first < 65535 ? tokens - first : 65535;
        const dim3 grid((width + 255) / 256 < 8 ? (width + 255) / 256 : 8, count);
        if (((width | x_stride | gate_stride | gate_off) & 3) == 0 && ((uintptr_t)gate & 15) == 0 && ((uintptr_t)x & (is_bf16 ? 7 : 15)) == 0) {
            const dim3 fours((width / 4 + 255) / 256, count);
            if (is_bf16)
                sigmoid_gate4_kernel<<<fours, 256, 0, stream>>>((__nv_bfloat16*)x + (size_t)first * x_stride, x_stride, gate + (size_t)first * gate_stride, gate_stride, gate_off,
                                                                scale, width);
            else
                sigmoid_gate4_kernel<<<fours, 256, 0, stream>>>((float*)x + (size_t)first * x_stride, x_stride, gate + (size_t)first * gate_stride, gate_stride, gate_off, scale, width);
            continue;
        }
        if (is_bf16)
            sigmoid_gate_kernel<<<grid, 256, 0, stream>>>((__nv_bfloat16*)x + (size_t)first * x_stride, x_stride, gate + (size_t)first * gate_stride, gate_stride,
                                                          gate_off, scale, width);
        else
            sigmoid_gate_kernel<<<grid, 256, 0, stream>>>((float*)x + (size_t)first * x_stride, x_stride, gate + (size_t)first * gate_stride, gate_stride, gate_off,
                                                          scale, width);
    }
    return launch_status();
}

// ---------------------------------------------------------------- residual add of up to two sublayer outputs + RMS norm in groups
// Output row r reads source row s = rows ? rows[r] : r:  v = h[s] + (d1[s] + d2[s]) (either may be absent; the two outputs are added
// to one another first, then to the stream), written back into h with `write_h`.  The row is cut into `groups` equal consecutive parts
// and each is divided by its own sqrt(mean(part^2) + eps); the whole is multiplied by the weight.  A warp owns a part's sum at a time
// (lanes stride over the part, then a butterfly), so the sums have one shape whatever the launch.  Everything is float until the one
// rounding of the result.  The row's sums are kept in shared memory (at most 64 groups).
template <typename TD, typename TO>
__global__ void __launch_bounds__(256) add_group_rmsnorm_kernel(float* __restrict__ h, const TD* __restrict__ d1, const TD* __restrict__ d2,
                                                                const float* __restrict__ weight, TO* __restrict__ out, const int* __restrict__ rows,
                                                                int hidden, int groups, float eps, int write_h) {
    __shared__ float inv[64];
    const int r = blockIdx.x;
    const int s = rows ? rows[r] : r;
    float* hrow = h + (size_t)s * hidden;
    const TD* a = d1 ? d1 + (size_t)s * hidden : nullptr;
    const TD* b = d2 ? d2 + (size_t)s * hidden : nullptr;
    const int part = hidden / groups, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    for (int g = warp; g < groups; g += warps) {
        float sum = 0.f;
        for (int i = g * part + lane; i < (g + 1) * part; i += 32) {
            float v = hrow[i];
            if (a && b) v += to_float(a[i]) + to_float(b[i]);
            else if (a) v += to_float(a[i]);
            else if (b) v += to_float(b[i]);
            if (write_h && (a || b)) hrow[i] = v;
            sum = fmaf(v, v, sum);
        }
        sum = warp_sum(sum);
        if (lane == 0) inv[g] = 1.0f / sqrtf(sum / (float)part + eps);
    }
    __syncthreads();
    TO* orow = out + (size_t)r * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        float v = hrow[i];
        if (!write_h) {
            if (a && b) v += to_float(a[i]) + to_float(b[i]);
            else if (a) v += to_float(a[i]);
            else if (b) v += to_float(b[i]);
        }
        orow[i] = from_float<TO>(v * inv[i / part] * weight[i]);
    }
}

// The same with four columns per access, for parts that are a multiple of four columns.  When the block has more warps than the row
// has groups, a group's columns are cut into equal runs, one per warp, and the runs' sums are added in order: the sums have one shape
// for a given row length and number of groups, whatever else is in the launch.
template <typename TD, typename TO>
__global__ void __launch_bounds__(512) add_group_rmsnorm4_kernel(float* __restrict__ h, const TD* __restrict__ d1, const TD* __restrict__ d2,
                                                                 const float* __restrict__ weight, TO* __restrict__ out, const int* __restrict__ rows,
                                                                 int hidden, int groups, float eps, int write_h) {
    __shared__ float inv[64], partial[64];
    const int r = blockIdx.x;
    const int s = rows ? rows[r] : r;
    float* hrow = h + (size_t)s * hidden;
    const TD* a = d1 ? d1 + (size_t)s * hidden : nullptr;
    const TD* b = d2 ? d2 + (size_t)s * hidden : nullptr;
    const int part = hidden / groups, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int runs = groups < warps ? warps / groups : 1, quads = part / 4, per_run = (quads + runs - 1) / runs;
    for (int item = warp; item < groups * runs; item += warps) {
        const int g = item / runs, k = item - g * runs;
        const int lo = g * part + min(quads, k * per_run) * 4, hi = g * part + min(quads, (k + 1) * per_run) * 4;
        float sum = 0.f;
#pragma unroll 4
        for (int i = lo + lane * 4; i < hi; i += 128) {
            float v[4], x[4];
            load4(hrow + i, v);
            if (a) {
                load4(a + i, x);
                if (b) {
                    float y[4];
                    load4(b + i, y);
#pragma unroll
                    for (int e = 0; e < 4; ++e) x[e] += y[e];
                }
            } else if (b) {
                load4(b + i, x);
            }
            if (a || b) {
#pragma unroll
                for (int e = 0; e < 4; ++e) v[e] += x[e];
                if (write_h) store4(hrow + i, v);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) sum = fmaf(v[e], v[e], sum);
        }
        sum = warp_sum(sum);
        if (lane == 0) partial[item] = sum;
    }
    __syncthreads();
    if (threadIdx.x < groups) {
        float sum = 0.f;
        for (int k = 0; k < runs; ++k) sum += partial[threadIdx.x * runs + k];
        inv[threadIdx.x] = 1.0f / sqrtf(sum / (float)part + eps);
    }
    __syncthreads();
    TO* orow = out + (size_t)r * hidden;
#pragma unroll 2
    for (int i = threadIdx.x * 4; i < hidden; i += blockDim.x * 4) {
        float v[4], w[4];
        load4(hrow + i, v);
        if (!write_h && (a || b)) {
            float x[4];
            if (a) {
                load4(a + i, x);
                if (b) {
                    float y[4];
                    load4(b + i, y);
#pragma unroll
                    for (int e = 0; e < 4; ++e) x[e] += y[e];
                }
            } else {
                load4(b + i, x);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] += x[e];
        }
        load4(weight + i, w);
        const float scale = inv[i / part];
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = v[e] * scale * w[e];
        store4(orow + i, v);
    }
}

HB_EXPORT int hb_add_group_rmsnorm(float* h, const void* d1, const void* d2, int delta_is_bf16, const float* weight, void* out, int out_is_bf16,
                                   const int* rows, int n_rows, int hidden, int groups, float eps, int write_h, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (hidden <= 0 || groups <= 0 || groups > 64 || hidden % groups) return HB_UNSUPPORTED_SIZE;
    const int threads = groups >= 8 ? 256 : (groups * 32 < 128 ? 128 : groups * 32);
    const bool by_four = (hidden / groups) % 4 == 0 && (((uintptr_t)h | (uintptr_t)d1 | (uintptr_t)d2 | (uintptr_t)weight | (uintptr_t)out) % 16) == 0;
#define HB_GROUP_NORM(TD, TO)                                                                                                                          \
    if (by_four) add_group_rmsnorm4_kernel<TD, TO><<<n_rows, hidden >= 4096 ? 512 : 256, 0, stream>>>(h, (const TD*)d1, (const TD*)d2, weight, (TO*)out, rows, hidden, groups, eps, write_h); \
    else add_group_rmsnorm_kernel<TD, TO><<<n_rows, threads, 0, stream>>>(h, (const TD*)d1, (const TD*)d2, weight, (TO*)out, rows, hidden, groups, eps, write_h)
    if (delta_is_bf16 && out_is_bf16) { HB_GROUP_NORM(__nv_bfloat16, __nv_bfloat16); }
    else if (delta_is_bf16) { HB_GROUP_NORM(__nv_bfloat16, float); }
    else if (out_is_bf16) { HB_GROUP_NORM(float, __nv_bfloat16); }
    else { HB_GROUP_NORM(float, float); }
#undef HB_GROUP_NORM
    return launch_status();
}

// ---------------------------------------------------------------- a gated unit whose gate and value are clamped
// in: [tokens, 2*inter], all gate columns first.  g = min(gate, limit); u = clamp(up, -limit, limit);
// out[t, i] = g * sigmoid(slope * g) * (u + 1), in float, rounded once.
template <typename T>
__global__ void clamped_glu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int inter, float limit, float slope) {
    const int t = blockIdx.y;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < inter; i += gridDim.x * blockDim.x) {
        const size_t at = (size_t)t * 2 * inter + i;
        const float g = fminf(to_float(gate_up[at]), limit);
        const float u = fminf(fmaxf(to_float(gate_up[at + inter]), -limit), limit);
        out[(size_t)t * inter + i] = from_float<T>(g / (1.0f + expf(-slope * g)) * (u + 1.0f));
    }
}

template <typename T>
__global__ void clamped_glu4_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int inter, float limit, float slope) {
    const int t = blockIdx.y;
    for (int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4; i < inter; i += gridDim.x * blockDim.x * 4) {
        const size_t at = (size_t)t * 2 * inter + i;
        float g[4], u[4];
        load4(gate_up + at, g);
        load4(gate_up + at + inter, u);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float gg = fminf(g[e], limit), uu = fminf(fmaxf(u[e], -limit), limit);
            g[e] = gg / (1.0f + expf(-slope * gg)) * (uu + 1.0f);
        }
        store4(out + (size_t)t * inter + i, g);
    }
}

HB_EXPORT int hb_clamped_glu(const void* gate_up, void* out, int is_bf16, int tokens, int inter, float limit, float slope, cudaStream_t stream) {
    if (tokens <= 0 || inter <= 0) return 0;
    const bool by_four = inter % 4 == 0 && (((uintptr_t)gate_up | (uintptr_t)out) % 16) == 0;
    for (int first = 0; first < tokens; first += 65535) {
        const int count = tokens - first < 65535 ? tokens - first : 65535;
        const int across = by_four ? (inter / 4 + 255) / 256 : (inter + 255) / 256;
        const dim3 grid(across < 16 ? across : 16, count);
#define HB_CLAMPED(T)                                                                                                                              \
    if (by_four) clamped_glu4_kernel<<<grid, 256, 0, stream>>>((const T*)gate_up + (size_t)first * 2 * inter, (T*)out + (size_t)first * inter, inter, limit, slope); \
    else clamped_glu_kernel<<<grid, 256, 0, stream>>>((const T*)gate_up + (size_t)first * 2 * inter, (T*)out + (size_t)first * inter, inter, limit, slope)
        if (is_bf16) { HB_CLAMPED(__nv_bfloat16); }
        else { HB_CLAMPED(float); }
#undef HB_CLAMPED
    }
    return launch_status();
}

// ---------------------------------------------------------------- GELU in its exact form, and a scale in place
// out = 0.5 z (1 + erf(z / sqrt(2))), in float, rounded once.  hb_scale_rows: x <- x * scale over a dense float tensor.
template <typename T>
__global__ void gelu_erf_kernel(const T* __restrict__ x, T* __restrict__ out, size_t count) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (size_t)gridDim.x * blockDim.x) {
        const float z = to_float(x[i]);
        out[i] = from_float<T>(0.5f * z * (1.f + erff(z * 0.7071067811865476f)));
    }
}

HB_EXPORT int hb_gelu_erf(const void* x, void* out, int is_bf16, long long count, cudaStream_t stream) {
    if (count <= 0) return 0;
    const int blocks = (int)((count + 255) / 256 < 8192 ? (count + 255) / 256 : 8192);
    if (is_bf16) gelu_erf_kernel<<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)x, (__nv_bfloat16*)out, (size_t)count);
    else gelu_erf_kernel<<<blocks, 256, 0, stream>>>((const float*)x, (float*)out, (size_t)count);
    return launch_status();
}

__global__ void scale_rows_kernel(float* __restrict__ x, float scale, size_t count) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (size_t)gridDim.x * blockDim.x) x[i] *= scale;
}

HB_EXPORT int hb_scale_rows(float* x, float scale, long long count, cudaStream_t stream) {
    if (count <= 0) return 0;
    const int blocks = (int)((count + 255) / 256 < 8192 ? (count + 255) / 256 : 8192);
    scale_rows_kernel<<<blocks, 256, 0, stream>>>(x, scale, (size_t)count);
    return launch_status();
}

// ---------------------------------------------------------------- the sum of two sublayers, then one norm or two of the same stream
// h <- h + (a + b) in the float stream, then out1 = h / sqrt(mean(h^2) + eps) * w1 and, where a second weight is given, out2 likewise with w2: two
// sublayers that read the same stream through norms of their own share its root mean square.  `a` is dense, or a product still in its split-K
// pieces (float, added up in split order); `b` is dense, or rows sorted by expert of which a token takes `top` with a weight each (added
// in the order of the choices).  With `rows` only those rows are worked on and h stays as it was.  Everything is float until the
// rounding of a result.  A row stays in the block's registers between the sum and the norm.
struct PairInputs {
    const void* a;          // [tokens, hidden], or float [splits, tokens, hidden] when a_splits > 0
    int a_splits;
    size_t a_split_stride;
    const void* b;          // [tokens, hidden], or [slots, hidden] when slot_of is given
    const int* slot_of;     // [tokens, top]
    const float* weights;   // [tokens, top]
    int top;
};

template <typename TD, int VEC>
__device__ __forceinline__ void read_entries(const TD* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) load4(p, v);
    else v[0] = to_float(p[0]);
}

template <typename TD, typename TO, int VEC, int CHUNKS>
__global__ void __launch_bounds__(512) add_pair_norms_kernel(float* __restrict__ h, const PairInputs in, const float* __restrict__ w1, const float* __restrict__ w2,
                                                             TO* __restrict__ out1, TO* __restrict__ out2, const int* __restrict__ rows, int hidden, float eps,
                                                             int write_h) {
    __shared__ float scratch[32];
    const int r = blockIdx.x, step = blockDim.x * VEC;
    float weight1[CHUNKS][VEC];
    let_next_kernel_start();
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {  // no kernel writes weights: these loads overlap the kernel before
        const int i = c * step + threadIdx.x * VEC;
        if (i < hidden) read_entries<float, VEC>(w1 + i, weight1[c]);
    }
    wait_for_previous_kernels();
    const int s = rows ? rows[r] : r;
    float* hrow = h + (size_t)s * hidden;
    float v[CHUNKS][VEC];
    float sum = 0.f;
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = c * step + threadIdx.x * VEC;
        if (i >= hidden) continue;
        read_entries<float, VEC>(hrow + i, v[c]);
        float add[VEC], x[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) add[e] = 0.f;
        if (in.a_splits > 0) {
            const float* p = (const float*)in.a + (size_t)s * hidden + i;
#pragma unroll 4
            for (int k = 0; k < in.a_splits; ++k) {
                read_entries<float, VEC>(p + (size_t)k * in.a_split_stride, x);
#pragma unroll
                for (int e = 0; e < VEC; ++e) add[e] += x[e];
            }
        } else if (in.a) {
            read_entries<TD, VEC>((const TD*)in.a + (size_t)s * hidden + i, add);
        }
        if (in.slot_of) {
            float fed[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) fed[e] = 0.f;
#pragma unroll 4
            for (int k = 0; k < in.top; ++k) {
                const int slot = in.slot_of[(size_t)s * in.top + k];
                const float w = in.weights[(size_t)s * in.top + k];
                if (slot < 0) continue;
                read_entries<TD, VEC>((const TD*)in.b + (size_t)slot * hidden + i, x);
#pragma unroll
                for (int e = 0; e < VEC; ++e) fed[e] = fmaf(w, x[e], fed[e]);
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) add[e] += fed[e];
        } else if (in.b) {
            read_entries<TD, VEC>((const TD*)in.b + (size_t)s * hidden + i, x);
#pragma unroll
            for (int e = 0; e < VEC; ++e) add[e] += x[e];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[c][e] += add[e];
        if (write_h && (in.a || in.b)) {
            if constexpr (VEC == 4) store4(hrow + i, v[c]);
            else hrow[i] = v[c][0];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) sum = fmaf(v[c][e], v[c][e], sum);
    }
    const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps);
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = c * step + threadIdx.x * VEC;
        if (i >= hidden) continue;
        float o[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = v[c][e] * inv * weight1[c][e];
        if constexpr (VEC == 4) store4(out1 + (size_t)r * hidden + i, o);
        else out1[(size_t)r * hidden + i] = from_float<TO>(o[0]);
        if (w2) {
            float w[VEC];
            read_entries<float, VEC>(w2 + i, w);
#pragma unroll
            for (int e = 0; e < VEC; ++e) o[e] = v[c][e] * inv * w[e];
            if constexpr (VEC == 4) store4(out2 + (size_t)r * hidden + i, o);
            else out2[(size_t)r * hidden + i] = from_float<TO>(o[0]);
        }
    }
}

// Rows that are no multiple of four entries (or not aligned to them) may have up to 4,096, others up to 16,384; bfloat16 sublayer outputs go with
// bfloat16 results.
HB_EXPORT int hb_add_pair_norms(float* h, const void* a, int a_splits, long long a_split_stride, const void* b, const int* slot_of, const float* weights, int top,
                                int delta_is_bf16, const float* w1, const float* w2, void* out1, void* out2, int out_is_bf16, const int* rows, int n_rows,
                                int hidden, float eps, int write_h, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (!w1 || !out1 || (w2 && !out2) || (slot_of && (!b || !weights || top <= 0)) || (a_splits > 0 && !a)) return HB_BAD_ARGUMENT;
    if (hidden <= 0 || hidden > 512 * 32 || (delta_is_bf16 && !out_is_bf16)) return HB_UNSUPPORTED_SIZE;
    const uintptr_t all = (uintptr_t)h | (uintptr_t)a | (uintptr_t)b | (uintptr_t)w1 | (uintptr_t)w2 | (uintptr_t)out1 | (uintptr_t)out2;
    const bool by_four = hidden % 4 == 0 && (all & 15) == 0 && (a_split_stride & 3) == 0;
    const PairInputs in{a, a_splits, (size_t)a_split_stride, b, slot_of, weights, top};
    const int pieces = by_four ? hidden / 4 : hidden;
    // the block's size and a thread's share follow from the row alone, so a row's sum has one shape whatever else is in the launch
    const int threads = pieces <= 128 ? 128 : (pieces <= 512 ? 256 : 512), chunks = (pieces + threads - 1) / threads;
#define HB_PAIR_LAUNCH(TD, TO, VEC, CHUNKS)                                                                                                                   \
    return launch_after_previous(add_pair_norms_kernel<TD, TO, VEC, CHUNKS>, dim3(n_rows), dim3(threads), 0, stream, h, in, w1, w2, (TO*)out1, (TO*)out2, rows, \
                                 hidden, eps, write_h)
#define HB_PAIR(TD, TO)                                    \
    if (by_four) {                                         \
        if (chunks <= 2) HB_PAIR_LAUNCH(TD, TO, 4, 2);     \
        HB_PAIR_LAUNCH(TD, TO, 4, 8);                      \
    }                                                      \
    if (chunks <= 2) HB_PAIR_LAUNCH(TD, TO, 1, 2);         \
    if (chunks > 8) return HB_UNSUPPORTED_SIZE;            \
    HB_PAIR_LAUNCH(TD, TO, 1, 8)
    if (delta_is_bf16 && out_is_bf16) { HB_PAIR(__nv_bfloat16, __nv_bfloat16); }
    if (out_is_bf16) { HB_PAIR(float, __nv_bfloat16); }
    HB_PAIR(float, float);
#undef HB_PAIR
#undef HB_PAIR_LAUNCH
}

// ---------------------------------------------------------------- a smooth cap in place
// x <- cap * tanh(x / cap) over a dense float tensor.
__global__ void soft_cap_kernel(float* __restrict__ x, float cap, size_t count) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4; i < count; i += (size_t)gridDim.x * blockDim.x * 4) {
        if (i + 4 <= count) {
            float v[4];
            load4(x + i, v);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = cap * tanhf(v[e] / cap);
            store4(x + i, v);
        } else {
            for (size_t j = i; j < count; ++j) x[j] = cap * tanhf(x[j] / cap);
        }
    }
}

HB_EXPORT int hb_soft_cap(float* x, float cap, long long count, cudaStream_t stream) {
    if (count <= 0) return 0;
    if (!(cap > 0.f) || ((uintptr_t)x & 15)) return HB_BAD_ARGUMENT;
    const long long blocks = (count + 1023) / 1024;
    return launch_after_previous(soft_cap_kernel, dim3((unsigned)(blocks < 8192 ? blocks : 8192)), dim3(256), 0, stream, x, cap, (size_t)count);
}

// ---------------------------------------------------------------- the square of relu
// out = max(z, 0)^2, in float, rounded once.
template <typename T>
__global__ void relu_squared_kernel(const T* __restrict__ x, T* __restrict__ out, size_t count) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (size_t)gridDim.x * blockDim.x)
        out[i] = from_float<T>(activated(to_float(x[i]), HB_ACT_RELU_SQUARED));
}

// Eight entries per thread and access, for 16-byte aligned tensors of a multiple of eight entries.
__global__ void relu_squared_bf16x8_kernel(const uint4* __restrict__ x, uint4* __restrict__ out, size_t eights) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < eights; i += (size_t)gridDim.x * blockDim.x) {
        uint4 raw = x[i];
        __nv_bfloat162* pairs = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(pairs[k]);
            pairs[k] = __floats2bfloat162_rn(activated(f.x, HB_ACT_RELU_SQUARED), activated(f.y, HB_ACT_RELU_SQUARED));
        }
        out[i] = raw;
    }
}

// The same of a product still in its split-K pieces ([splits, count] floats, added up in split order): what would add them up applies the activation at once.
template <typename T>
__global__ void relu_squared_of_pieces_kernel(const float* __restrict__ pieces, int splits, size_t count, T* __restrict__ out) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4; i < count; i += (size_t)gridDim.x * blockDim.x * 4) {
        float sum[4] = {0.f, 0.f, 0.f, 0.f}, piece[4];
#pragma unroll 8
        for (int k = 0; k < splits; ++k) {
            load4(pieces + (size_t)k * count + i, piece);
#pragma unroll
            for (int e = 0; e < 4; ++e) sum[e] += piece[e];
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) sum[e] = activated(sum[e], HB_ACT_RELU_SQUARED);
        store4(out + i, sum);
    }
}

HB_EXPORT int hb_relu_squared_of_pieces(const float* pieces, int splits, long long count, void* out, int out_is_bf16, cudaStream_t stream) {
    if (count <= 0) return 0;
    if (splits < 1 || count % 4 || (((uintptr_t)pieces | (uintptr_t)out) & 15)) return HB_UNSUPPORTED_SIZE;
    const long long wanted = (count / 4 + 127) / 128;
    const dim3 blocks((unsigned)(wanted < 16384 ? wanted : 16384));
    if (out_is_bf16) return launch_after_previous(relu_squared_of_pieces_kernel<__nv_bfloat16>, blocks, dim3(128), 0, stream, pieces, splits, (size_t)count, (__nv_bfloat16*)out);
    return launch_after_previous(relu_squared_of_pieces_kernel<float>, blocks, dim3(128), 0, stream, pieces, splits, (size_t)count, (float*)out);
}

HB_EXPORT int hb_relu_squared(const void* x, void* out, int is_bf16, long long count, cudaStream_t stream) {
    if (count <= 0) return 0;
    const bool eights = is_bf16 && count % 8 == 0 && (((uintptr_t)x | (uintptr_t)out) & 15) == 0;
    const long long items = eights ? count / 8 : count, wanted = (items + 255) / 256;
    const dim3 blocks((unsigned)(wanted < 16384 ? wanted : 16384));
    if (eights) return launch_after_previous(relu_squared_bf16x8_kernel, blocks, dim3(256), 0, stream, (const uint4*)x, (uint4*)out, (size_t)items);
    if (is_bf16) return launch_after_previous(relu_squared_kernel<__nv_bfloat16>, blocks, dim3(256), 0, stream, (const __nv_bfloat16*)x, (__nv_bfloat16*)out, (size_t)count);
    return launch_after_previous(relu_squared_kernel<float>, blocks, dim3(256), 0, stream, (const float*)x, (float*)out, (size_t)count);
}
