// Recurrences whose matrix state fades by one number per token and head, walked in chunks of 64 tokens on the tensor cores:
//     S <- a_t S + b_t k_t v_t^T;   o_t = S^T q_t                     (the state-space recurrence, a matrix memory, retention)
// With L_t the sum of ln a up to token t of its chunk and S0 the state at the chunk's start,
//     o_i = exp(L_i) S0^T q_i + sum_(j <= i) exp(L_i - L_j) b_j (q_i . k_j) v_j,
//     S_end = exp(L_end) S0 + sum_j exp(L_end - L_j) b_j k_j v_j^T,
// so chunks need one another only through S0: chunk_states makes every chunk's own sum (the second line without S0) and its decay exp(L_end),
// chunk_join walks the short chain per state entry, and chunk_outputs makes the outputs.  Products run as mma.sync with float sums.  Keys, queries and
// values, which are projections, are rounded to bfloat16; everything else is float: logarithms, decays, steps and the state, and where one of them is an operand
// of a product (weighted scores, weighted values, the state) it enters as a bfloat16 and a bfloat16 remainder, 16 bits of it, in two products.
// A matrix memory also sums its keys, n <- a n + b k: the state's row behind the values; n . q is the plain sum of a row's weighted scores
// plus exp(L_i) n0 . q_i.  The one-token-after-another form of the same recurrences (recurrent.cu) serves decoded tokens and the float32 mode.
// A block takes ETILE value columns of one head and chunk (64, or 128 where a head has them) with two threads per column.
#include "common.cuh"

namespace {
constexpr int CHUNK = 64, AHEAD = 8;  // AHEAD: 16-byte loads a thread has on their way at once
enum : int { KIND_STATE_SPACE = 0, KIND_GIVEN = 1 };

struct ChunkArgs {
    const float* k;      // [tokens, stride]: group g at g * n
    const float* q;
    const float* v;      // head h at h * e
    int k_stride, q_stride, v_stride;
    const float* gate;   // state space: the step's pre-activation of head h at decay_off + h; given: ln of the decay at decay_off + h, the step at step_off + h
    int gate_stride, decay_off, step_off;
    const float* a_log;  // [heads] (state space)
    const float* dt_bias;
    const float* skip;   // [heads] (state space: D)
    float* ends;         // [chunks, end_stride]: head h at h * (e + sums) * n_padded, [e (+ 1), n_padded]
    size_t end_stride;
    float* decays;       // [chunks, heads]
    __nv_bfloat16* begins;  // [chunks, heads, e (+ 1), 2, n16]: the state at every chunk's start, its rounded value and the remainder (n16: n up to a multiple of 16)
    const int* start;    // [chunks + 1]: the first token of every chunk (chunks are consecutive)
    float* out;          // [tokens, heads, out_e]
    int out_e;
    int heads, groups, n, n_padded, e;
    int sums;            // 1: the state has a row for the sum of keys
    float q_scale;
    int by_four;         // columns and strides allow 16-byte loads
    int by_two;          // outputs may be stored in pairs
};

__device__ __forceinline__ float softplus_of(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// L[j] (the running sum of log2 a) and the step of every token of the chunk (threads 0 .. 63 of the block); past the end: L stays, step 0.
template <int KIND>
__device__ __forceinline__ void chunk_gates(const ChunkArgs& a, int first, int count, int head, float* L, float* step, float* warp_total) {
    const int j = threadIdx.x, lane = j & 31;
    float log_decay = 0.f, b = 0.f;
    if (j < count) {
        const float* g = a.gate + (size_t)(first + j) * a.gate_stride;
        if (KIND == KIND_STATE_SPACE) {
            b = softplus_of(g[a.decay_off + head] + a.dt_bias[head]);
            log_decay = -expf(a.a_log[head]) * b;
        } else {
            log_decay = g[a.decay_off + head];
            b = g[a.step_off + head];
        }
    }
    float sum = log_decay;
    if (j < CHUNK) {
#pragma unroll
        for (int offset = 1; offset < 32; offset <<= 1) {
            const float other = __shfl_up_sync(0xffffffffu, sum, offset);
            if (lane >= offset) sum += other;
        }
        if (j == 31) *warp_total = sum;
    }
    __syncthreads();
    if (j < CHUNK) {
        L[j] = (j >= 32 ? sum + *warp_total : sum) * 1.4426950408889634f;
        step[j] = b;
    }
    __syncthreads();
}

__device__ __forceinline__ uint32_t pack(float lo, float hi) {
    const __nv_bfloat162 both = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&both);
}

// Two floats as bfloat16 and what that rounding left of them.
__device__ __forceinline__ void pack_pair(float a, float b, uint32_t& rounded, uint32_t& rest) {
    const __nv_bfloat162 both = __floats2bfloat162_rn(a, b);
    rounded = *reinterpret_cast<const uint32_t*>(&both);
    rest = pack(a - __low2float(both), b - __high2float(both));
}

// A tile of CHUNK rows of floats on its way to shared memory as bfloat16: row r at src + r * stride; rows from `live` on and columns from `columns` on are zeros.
// fetch() asks for AHEAD pieces of four columns from piece `base` on; place() rounds them, times `factor`, into rows of `ld` columns.
struct Tile {
    const float* src;
    size_t stride;
    int live, columns, quads;  // quads: pieces per row
    bool by_four;

    // a walk over the tile's pieces in steps of THREADS without a division per piece
    template <int THREADS>
    struct Walk {
        int r, quad, rows, rest, quads;
        __device__ __forceinline__ Walk(int first, int quads_) : r(first / quads_), quad(first % quads_), rows(THREADS / quads_), rest(THREADS % quads_), quads(quads_) {}
        __device__ __forceinline__ void next() {
            r += rows;
            quad += rest;
            if (quad >= quads) { quad -= quads; ++r; }
        }
    };

    template <int THREADS>
    __device__ __forceinline__ void fetch(Walk<THREADS> at, float (&x)[AHEAD][4]) const {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u, at.next()) {
            x[u][0] = x[u][1] = x[u][2] = x[u][3] = 0.f;
            const int c = at.quad * 4;
            if (at.r < live) {
                const float* p = src + (size_t)at.r * stride + c;
                if (by_four && c + 4 <= columns) {
                    load4(p, x[u]);
                } else {
#pragma unroll
                    for (int i = 0; i < 4; ++i) x[u][i] = c + i < columns ? p[i] : 0.f;
                }
            }
        }
    }

    template <int THREADS>
    __device__ __forceinline__ void place(Walk<THREADS> at, const float (&x)[AHEAD][4], __nv_bfloat16* dst, int ld, float factor) const {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u, at.next()) {
            if (at.r >= CHUNK) continue;
            uint2 packed;
            packed.x = pack(x[u][0] * factor, x[u][1] * factor);
            packed.y = pack(x[u][2] * factor, x[u][3] * factor);
            *reinterpret_cast<uint2*>(dst + at.r * ld + at.quad * 4) = packed;
        }
    }

    // rows times a float each: the rounded value and the remainder
    template <int THREADS>
    __device__ __forceinline__ void place_weighted(Walk<THREADS> at, const float (&x)[AHEAD][4], __nv_bfloat16* hi, __nv_bfloat16* lo, int ld, const float* row_factor) const {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u, at.next()) {
            if (at.r >= CHUNK) continue;
            const float f = row_factor[at.r];
            uint2 rounded, rest;
            pack_pair(x[u][0] * f, x[u][1] * f, rounded.x, rest.x);
            pack_pair(x[u][2] * f, x[u][3] * f, rounded.y, rest.y);
            *reinterpret_cast<uint2*>(hi + at.r * ld + at.quad * 4) = rounded;
            *reinterpret_cast<uint2*>(lo + at.r * ld + at.quad * 4) = rest;
        }
    }
};

__device__ __forceinline__ uint32_t shared_address(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void load_matrices(uint32_t (&r)[4], uint32_t address) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address));
}
__device__ __forceinline__ void load_matrices_turned(uint32_t (&r)[4], uint32_t address) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address));
}
__device__ __forceinline__ void multiply(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// What a chunk adds to the state: grid (chunks, heads, tiles of value columns); warp w owns 16 of the tile's columns (rows of S^T).
template <int KIND, int NMAX, int ETILE>
__global__ void __launch_bounds__(2 * ETILE) chunk_states_kernel(const ChunkArgs a) {
    constexpr int THREADS = 2 * ETILE;
    extern __shared__ __align__(16) unsigned char memory[];
    __shared__ __align__(16) float L[CHUNK], step[CHUNK], warp_total;
    const int chunk = blockIdx.x, head = blockIdx.y, e0 = blockIdx.z * ETILE;
    const int first = a.start[chunk], count = a.start[chunk + 1] - first;
    const int n16 = (a.n + 15) & ~15, k_ld = n16 + 8;
    constexpr int v_ld = ETILE + 8;
    __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(memory);
    __nv_bfloat16* vs = ks + CHUNK * k_ld;
    __nv_bfloat16* vs_rest = vs + CHUNK * v_ld;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int group = head / (a.heads / a.groups);

    const Tile keys{a.k + (size_t)first * a.k_stride + (size_t)group * a.n, (size_t)a.k_stride, count, a.n, n16 / 4, a.by_four != 0};
    const Tile values{a.v + (size_t)first * a.v_stride + (size_t)head * a.e + e0, (size_t)a.v_stride, count, min(ETILE, a.e - e0), ETILE / 4, a.by_four != 0};
    const Tile::Walk<THREADS> key_walk(threadIdx.x, keys.quads), value_walk(threadIdx.x, ETILE / 4);
    float x[AHEAD][4], y[AHEAD][4];
    keys.fetch(key_walk, x);
    values.fetch(value_walk, y);  // AHEAD pieces per thread are the whole tile
    chunk_gates<KIND>(a, first, count, head, L, step, &warp_total);
    const float last = L[CHUNK - 1];
    if (threadIdx.x < CHUNK) step[threadIdx.x] *= exp2f(last - L[threadIdx.x]);  // the weight of a token in the chunk's sum
    if (threadIdx.x == 0 && blockIdx.z == 0) a.decays[(size_t)chunk * a.heads + head] = exp2f(last);
    keys.place(key_walk, x, ks, k_ld, 1.f);
    for (int base = threadIdx.x + AHEAD * THREADS; base < CHUNK * keys.quads; base += AHEAD * THREADS) {
        const Tile::Walk<THREADS> walk(base, keys.quads);
        keys.fetch(walk, x);
        keys.place(walk, x, ks, k_ld, 1.f);
    }
    __syncthreads();  // the weights are there
    values.place_weighted(value_walk, y, vs, vs_rest, v_ld, step);
    __syncthreads();

    float acc[NMAX / 8][4];
#pragma unroll
    for (int i = 0; i < NMAX / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int t = 0; t < CHUNK / 16; ++t) {
        uint32_t va[4], rest[4];  // rows: value columns; inner: tokens
        const int spot = (t * 16 + (lane >> 4) * 8 + (lane & 7)) * v_ld + warp * 16 + ((lane >> 3) & 1) * 8;
        load_matrices_turned(va, shared_address(vs + spot));
        load_matrices_turned(rest, shared_address(vs_rest + spot));
#pragma unroll
        for (int c = 0; c < NMAX / 16; ++c) {
            if (c * 16 >= n16) continue;
            uint32_t kb[4];
            load_matrices_turned(kb, shared_address(ks + (t * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * k_ld + c * 16 + (lane >> 4) * 8));
            multiply(acc[2 * c], va, kb[0], kb[1]);
            multiply(acc[2 * c + 1], va, kb[2], kb[3]);
            multiply(acc[2 * c], rest, kb[0], kb[1]);
            multiply(acc[2 * c + 1], rest, kb[2], kb[3]);
        }
    }
    float* dst = a.ends + (size_t)chunk * a.end_stride + (size_t)head * (a.e + a.sums) * a.n_padded;
#pragma unroll
    for (int i = 0; i < NMAX / 8; ++i) {
        const int column = i * 8 + (lane & 3) * 2;
        if (column >= a.n_padded) continue;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int row = e0 + warp * 16 + (lane >> 2) + half * 8;
            if (row < a.e) *reinterpret_cast<float2*>(dst + (size_t)row * a.n_padded + column) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
        }
    }
    if (a.sums && blockIdx.z == 0) {
        for (int c = threadIdx.x; c < a.n_padded; c += THREADS) {
            float sum = 0.f;
            if (c < a.n)
                for (int j = 0; j < count; ++j) sum = fmaf(step[j], __bfloat162float(ks[j * k_ld + c]), sum);
            dst[(size_t)a.e * a.n_padded + c] = sum;
        }
    }
}

// The chain through a row's chunks, two neighbouring state entries per thread: every chunk's start state to begins, the row's record ends up holding the
// state behind its last chunk.  Entries from n_padded on (up to n16) are zeros.
__global__ void chunk_join_kernel(const float* __restrict__ ends, size_t end_stride, const float* __restrict__ decays, __nv_bfloat16* __restrict__ begins, float* __restrict__ state,
                                  size_t slot_stride, int state_off, const int* __restrict__ slots, const int* __restrict__ chunk_row, int chunks, int heads, int rows, int n_padded,
                                  int n16) {
    const int pair = blockIdx.x * blockDim.x + threadIdx.x, pairs = n16 / 2;
    if (pair >= heads * rows * pairs) return;
    const int line = pair / pairs, column = (pair - line * pairs) * 2, head = line / rows;  // line: a row of a head's state
    const bool real = column < n_padded;
    const size_t from = (size_t)line * n_padded + column, to = (size_t)line * 2 * n16 + column, begin_stride = (size_t)heads * rows * 2 * n16;
    constexpr int AT_ONCE = 8;  // what the chunks add is asked for before the chain through them starts
    int j = 0;
    while (j < chunks) {
        const int row = chunk_row[j];
        float* kept = state + (size_t)slots[row] * slot_stride + state_off + from;
        float2 s = real ? *reinterpret_cast<const float2*>(kept) : make_float2(0.f, 0.f);
        while (j < chunks && chunk_row[j] == row) {
            float2 added[AT_ONCE];
            float fade[AT_ONCE];
            int count = 0;
#pragma unroll
            for (int k = 0; k < AT_ONCE; ++k) {
                if (j + k < chunks && chunk_row[j + k] == row) {
                    added[k] = real ? *reinterpret_cast<const float2*>(ends + (size_t)(j + k) * end_stride + from) : make_float2(0.f, 0.f);
                    fade[k] = decays[(size_t)(j + k) * heads + head];
                    count = k + 1;
                }
            }
#pragma unroll
            for (int k = 0; k < AT_ONCE; ++k) {
                if (k < count) {
                    __nv_bfloat16* dst = begins + (size_t)(j + k) * begin_stride + to;
                    const __nv_bfloat162 rounded = __floats2bfloat162_rn(s.x, s.y);
                    *reinterpret_cast<__nv_bfloat162*>(dst) = rounded;
                    *reinterpret_cast<__nv_bfloat162*>(dst + n16) = __floats2bfloat162_rn(s.x - __low2float(rounded), s.y - __high2float(rounded));
                    s.x = fmaf(fade[k], s.x, added[k].x);
                    s.y = fmaf(fade[k], s.y, added[k].y);
                }
            }
            j += count;
        }
        if (real) *reinterpret_cast<float2*>(kept) = s;
    }
}

__device__ __forceinline__ void copy_ahead(uint32_t to, const void* from, bool live) {  // 16 bytes, zeros where not live
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to), "l"(from), "r"(live ? 16 : 0));
}

// The outputs of a chunk from its start state: grid (chunks, heads, tiles of value columns); warp w owns tokens 16 (w % 4) .. + 15 and 64 of the tile's columns.
// First the queries meet the start state; then keys and values take the state's place in shared memory, which lets two blocks share an SM.
template <int KIND, int ETILE>
__global__ void __launch_bounds__(2 * ETILE, 256 / ETILE) chunk_outputs_kernel(const ChunkArgs a) {
    constexpr int THREADS = 2 * ETILE, COLUMNS = 64;
    extern __shared__ __align__(16) unsigned char memory[];
    __shared__ __align__(16) float L[CHUNK], step[CHUNK], warp_total;
    const int chunk = blockIdx.x, head = blockIdx.y, e0 = blockIdx.z * ETILE;
    const int first = a.start[chunk], count = a.start[chunk + 1] - first;
    const int n16 = (a.n + 15) & ~15, ld = n16 + 8;
    constexpr int v_ld = ETILE + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(memory);
    __nv_bfloat16* s_hi = qs + CHUNK * ld;
    __nv_bfloat16* s_lo = s_hi + ETILE * ld;
    __nv_bfloat16* ks = s_hi;  // CHUNK <= ETILE rows
    __nv_bfloat16* vs = ks + CHUNK * ld;
    const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3, column0 = (threadIdx.x >> 7) * COLUMNS;
    const int group = head / (a.heads / a.groups);
    const __nv_bfloat16* begin = a.begins + ((size_t)chunk * a.heads + head) * (a.e + a.sums) * 2 * n16;

    {
        const int pieces = n16 / 4;  // both halves of a state row lie side by side: n16 / 8 pieces of 16 bytes each
        Tile::Walk<THREADS> at(threadIdx.x, pieces);
        for (; at.r < ETILE; at.next()) {
            const int half = at.quad >= pieces / 2, c = (at.quad - half * (pieces / 2)) * 8;
            const bool live = e0 + at.r < a.e;
            copy_ahead(shared_address((half ? s_lo : s_hi) + at.r * ld + c), begin + (size_t)(live ? e0 + at.r : 0) * 2 * n16 + at.quad * 8, live);
        }
    }
    asm volatile("cp.async.commit_group;");
    const Tile queries{a.q + (size_t)first * a.q_stride + (size_t)group * a.n, (size_t)a.q_stride, count, a.n, n16 / 4, a.by_four != 0};
    const Tile keys{a.k + (size_t)first * a.k_stride + (size_t)group * a.n, (size_t)a.k_stride, count, a.n, n16 / 4, a.by_four != 0};
    const Tile values{a.v + (size_t)first * a.v_stride + (size_t)head * a.e + e0, (size_t)a.v_stride, count, min(ETILE, a.e - e0), ETILE / 4, a.by_four != 0};
    const Tile::Walk<THREADS> walk(threadIdx.x, n16 / 4), value_walk(threadIdx.x, ETILE / 4);
    float x[AHEAD][4], y[AHEAD][4];
    queries.fetch(walk, x);
    chunk_gates<KIND>(a, first, count, head, L, step, &warp_total);
    queries.place(walk, x, qs, ld, a.q_scale);
    for (int base = threadIdx.x + AHEAD * THREADS; base < CHUNK * queries.quads; base += AHEAD * THREADS) {
        const Tile::Walk<THREADS> more(base, queries.quads);
        queries.fetch(more, x);
        queries.place(more, x, qs, ld, a.q_scale);
    }
    asm volatile("cp.async.wait_all;");
    __syncthreads();

    const int row0 = warp * 16, g = lane >> 2, t2 = (lane & 3) * 2;
    const bool active = row0 < count;
    float acc[COLUMNS / 8][4];
#pragma unroll
    for (int i = 0; i < COLUMNS / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const int spot = ((lane >> 4) * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8;  // this lane's row of the four matrices of a step, rows n-major
    if (active) {
        for (int c = 0; c < n16; c += 16) {
            uint32_t qa[4];
            load_matrices(qa, shared_address(qs + (row0 + (lane & 15)) * ld + c + (lane >> 4) * 8));
#pragma unroll
            for (int i = 0; i < COLUMNS / 16; ++i) {
                uint32_t b[4];
                load_matrices(b, shared_address(s_hi + (column0 + i * 16) * ld + spot + c));
                multiply(acc[2 * i], qa, b[0], b[1]);
                multiply(acc[2 * i + 1], qa, b[2], b[3]);
                load_matrices(b, shared_address(s_lo + (column0 + i * 16) * ld + spot + c));
                multiply(acc[2 * i], qa, b[0], b[1]);
                multiply(acc[2 * i + 1], qa, b[2], b[3]);
            }
        }
    }
    keys.fetch(walk, x);
    values.fetch(value_walk, y);  // AHEAD pieces per thread are the whole tile
    __syncthreads();  // the state has been read
    keys.place(walk, x, ks, ld, 1.f);
    for (int base = threadIdx.x + AHEAD * THREADS; base < CHUNK * keys.quads; base += AHEAD * THREADS) {
        const Tile::Walk<THREADS> more(base, keys.quads);
        keys.fetch(more, x);
        keys.place(more, x, ks, ld, 1.f);
    }
    values.place(value_walk, y, vs, v_ld, 1.f);
    __syncthreads();
    if (active) {
        float score[CHUNK / 8][4];
#pragma unroll
        for (int i = 0; i < CHUNK / 8; ++i) score[i][0] = score[i][1] = score[i][2] = score[i][3] = 0.f;
        for (int c = 0; c < n16; c += 16) {
            uint32_t qa[4];
            load_matrices(qa, shared_address(qs + (row0 + (lane & 15)) * ld + c + (lane >> 4) * 8));
#pragma unroll
            for (int i = 0; i < CHUNK / 16; ++i) {
                if (i > warp) continue;  // keys behind every query of this warp
                uint32_t b[4];
                load_matrices(b, shared_address(ks + i * 16 * ld + spot + c));
                multiply(score[2 * i], qa, b[0], b[1]);
                multiply(score[2 * i + 1], qa, b[2], b[3]);
            }
        }
        const float top = L[row0 + g], bottom = L[row0 + g + 8];
        const float fade_top = exp2f(top), fade_bottom = exp2f(bottom);
#pragma unroll
        for (int i = 0; i < COLUMNS / 8; ++i) {
            acc[i][0] *= fade_top; acc[i][1] *= fade_top;
            acc[i][2] *= fade_bottom; acc[i][3] *= fade_bottom;
        }
        float sum_top = 0.f, sum_bottom = 0.f;
#pragma unroll
        for (int i = 0; i < CHUNK / 8; ++i) {
            if (i > 2 * warp + 1) continue;
            const float2 ahead = *reinterpret_cast<const float2*>(&L[i * 8 + t2]), weight = *reinterpret_cast<const float2*>(&step[i * 8 + t2]);
#pragma unroll
            for (int z = 0; z < 2; ++z) {
                const int j = i * 8 + t2 + z;
                const float l = z ? ahead.y : ahead.x, b = z ? weight.y : weight.x;
                score[i][z] = j <= row0 + g ? score[i][z] * (exp2f(top - l) * b) : 0.f;
                score[i][2 + z] = j <= row0 + g + 8 ? score[i][2 + z] * (exp2f(bottom - l) * b) : 0.f;
                sum_top += score[i][z];
                sum_bottom += score[i][2 + z];
            }
        }
#pragma unroll
        for (int i = 0; i < CHUNK / 16; ++i) {
            if (i > warp) continue;
            uint32_t pa[4], rest[4];
            pack_pair(score[2 * i][0], score[2 * i][1], pa[0], rest[0]);
            pack_pair(score[2 * i][2], score[2 * i][3], pa[1], rest[1]);
            pack_pair(score[2 * i + 1][0], score[2 * i + 1][1], pa[2], rest[2]);
            pack_pair(score[2 * i + 1][2], score[2 * i + 1][3], pa[3], rest[3]);
#pragma unroll
            for (int c = 0; c < COLUMNS / 16; ++c) {
                uint32_t b[4];
                load_matrices_turned(b, shared_address(vs + (i * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * v_ld + column0 + c * 16 + (lane >> 4) * 8));
                multiply(acc[2 * c], pa, b[0], b[1]);
                multiply(acc[2 * c + 1], pa, b[2], b[3]);
                multiply(acc[2 * c], rest, b[0], b[1]);
                multiply(acc[2 * c + 1], rest, b[2], b[3]);
            }
        }
        const float skip = KIND == KIND_STATE_SPACE ? a.skip[head] : 0.f;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int i = row0 + g + half * 8;
            if (i >= count) continue;
            float* dst = a.out + ((size_t)(first + i) * a.heads + head) * a.out_e + e0 + column0 + t2;
            const float* own = a.v + (size_t)(first + i) * a.v_stride + (size_t)head * a.e + e0 + column0 + t2;
            const int live = a.e - e0 - column0 - t2;  // entries from this lane's first one to the head's end
            float mine[COLUMNS / 8][2];
            if (KIND == KIND_STATE_SPACE) {
#pragma unroll
                for (int c = 0; c < COLUMNS / 8; ++c) {
#pragma unroll
                    for (int z = 0; z < 2; ++z) mine[c][z] = c * 8 + z < live ? skip * own[c * 8 + z] : 0.f;
                }
            }
#pragma unroll
            for (int c = 0; c < COLUMNS / 8; ++c) {
                float2 o = make_float2(acc[c][2 * half], acc[c][2 * half + 1]);
                if (KIND == KIND_STATE_SPACE) { o.x += mine[c][0]; o.y += mine[c][1]; }
                if (a.by_two && c * 8 + 1 < live) {
                    *reinterpret_cast<float2*>(dst + c * 8) = o;
                } else {
                    if (c * 8 < live) dst[c * 8] = o.x;
                    if (c * 8 + 1 < live) dst[c * 8 + 1] = o.y;
                }
            }
        }
        if (a.sums && blockIdx.z == 0 && column0 == 0) {  // n . q: a row's weighted scores, and what the chunk found
            sum_top += __shfl_xor_sync(0xffffffffu, sum_top, 1);
            sum_top += __shfl_xor_sync(0xffffffffu, sum_top, 2);
            sum_bottom += __shfl_xor_sync(0xffffffffu, sum_bottom, 1);
            sum_bottom += __shfl_xor_sync(0xffffffffu, sum_bottom, 2);
            const __nv_bfloat16* kept = begin + (size_t)a.e * 2 * n16;
            float found_top = 0.f, found_bottom = 0.f;
            for (int c = lane & 3; c < a.n; c += 4) {
                const float x = __bfloat162float(kept[c]) + __bfloat162float(kept[n16 + c]);
                found_top = fmaf(__bfloat162float(qs[(row0 + g) * ld + c]), x, found_top);
                found_bottom = fmaf(__bfloat162float(qs[(row0 + g + 8) * ld + c]), x, found_bottom);
            }
            found_top += __shfl_xor_sync(0xffffffffu, found_top, 1);
            found_top += __shfl_xor_sync(0xffffffffu, found_top, 2);
            found_bottom += __shfl_xor_sync(0xffffffffu, found_bottom, 1);
            found_bottom += __shfl_xor_sync(0xffffffffu, found_bottom, 2);
            if ((lane & 3) == 0) {
                if (row0 + g < count) a.out[((size_t)(first + row0 + g) * a.heads + head) * a.out_e + a.e] = fmaf(fade_top, found_top, sum_top);
                if (row0 + g + 8 < count) a.out[((size_t)(first + row0 + g + 8) * a.heads + head) * a.out_e + a.e] = fmaf(fade_bottom, found_bottom, sum_bottom);
            }
        }
    }
}

template <typename Kernel>
int allow_shared(Kernel kernel, int bytes) {
    return bytes > 48 * 1024 ? (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) : 0;
}

template <int KIND, int ETILE>
int launch_states(const ChunkArgs& a, int chunks, cudaStream_t stream) {
    const int n16 = (a.n + 15) & ~15, bytes = CHUNK * (n16 + 8) * 2 + 2 * CHUNK * (ETILE + 8) * 2;
    const dim3 grid(chunks, a.heads, (a.e + ETILE - 1) / ETILE);
#define HB_CHUNK_STATES(NMAX)                                                                        \
    do {                                                                                             \
        const int status = allow_shared(chunk_states_kernel<KIND, NMAX, ETILE>, bytes);              \
        if (status) return status;                                                                   \
        chunk_states_kernel<KIND, NMAX, ETILE><<<grid, 2 * ETILE, bytes, stream>>>(a);               \
    } while (0)
    if (n16 <= 64) HB_CHUNK_STATES(64);
    else if (n16 <= 128) HB_CHUNK_STATES(128);
    else HB_CHUNK_STATES(256);
#undef HB_CHUNK_STATES
    return launch_status();
}

template <int KIND, int ETILE>
int launch_outputs(const ChunkArgs& a, int chunks, cudaStream_t stream) {
    const int n16 = (a.n + 15) & ~15, state = 2 * ETILE * (n16 + 8) * 2, tiles = CHUNK * (n16 + 8) * 2 + CHUNK * (ETILE + 8) * 2, bytes = CHUNK * (n16 + 8) * 2 + (state > tiles ? state : tiles);
    const int status = allow_shared(chunk_outputs_kernel<KIND, ETILE>, bytes);
    if (status) return status;
    chunk_outputs_kernel<KIND, ETILE><<<dim3(chunks, a.heads, (a.e + ETILE - 1) / ETILE), 2 * ETILE, bytes, stream>>>(a);
    return launch_status();
}

template <int KIND>
int launch_chunks(const ChunkArgs& a, int chunks, float* state, long long slot_stride, int state_off, const int* slots, const int* chunk_row, cudaStream_t stream) {
    // 128 value columns to a block where a head has more than 64 and keys leave room for their states in shared memory
    const int n16 = (a.n + 15) & ~15, rows = a.e + a.sums;
    const bool wide = a.e > 64 && n16 <= 128;
    int status = wide ? launch_states<KIND, 128>(a, chunks, stream) : launch_states<KIND, 64>(a, chunks, stream);
    if (status) return status;
    const int pairs = a.heads * rows * (n16 / 2);
    chunk_join_kernel<<<(pairs + 127) / 128, 128, 0, stream>>>(a.ends, a.end_stride, a.decays, a.begins, state, (size_t)slot_stride, state_off, slots, chunk_row, chunks, a.heads, rows,
                                                             a.n_padded, n16);
    status = launch_status();
    if (status) return status;
    return wide ? launch_outputs<KIND, 128>(a, chunks, stream) : launch_outputs<KIND, 64>(a, chunks, stream);
}
}  // namespace

// The three passes over `chunks` chunks of at most 64 consecutive tokens (start [chunks + 1]; the chunks of a row follow one another, chunk_row names it).  kind 0: the
// state-space recurrence (step softplus(gate[decay_off + h] + dt_bias), ln decay = -exp(a_log) step, the value times skip added to the output); kind 1: ln decay and
// step given at decay_off + h and step_off + h of `gate`.  The state of (slot, head) is [e (+ 1 with sums), n_padded] floats at state + slot * slot_stride + state_off.
// Scratch: ends [chunks, heads * rows * n_padded] float, decays [chunks, heads] float, begins [chunks, heads, rows, 2, n16] bfloat16 with n16 = n up to a multiple of
// 16, rows = e + sums.  out [tokens, heads, out_e]; with sums (the state has a row behind its e value rows for the sum of keys) a head's entry e is n . q.
HB_EXPORT int hb_chunked_scan(int kind, const float* k, int k_stride, const float* q, int q_stride, const float* v, int v_stride, const float* gate, int gate_stride,
                              int decay_off, int step_off, const float* a_log, const float* dt_bias, const float* skip, float* ends, float* decays, void* begins, float* state,
                              long long slot_stride, int state_off, const int* slots, const int* start, const int* chunk_row, int chunks, float* out, int out_e, int heads,
                              int groups, int n, int n_padded, int e, int sums, float q_scale, cudaStream_t stream) {
    if (chunks <= 0) return 0;
    if (n <= 0 || n > 256 || e <= 0 || heads <= 0 || heads > 65535 || groups <= 0 || heads % groups || (e + 63) / 64 > 65535) return HB_UNSUPPORTED_SIZE;
    if (n_padded < n || n_padded - n > 3 || (n_padded & 3) || (slot_stride & 3) || (state_off & 3) || ((((uintptr_t)ends) | ((uintptr_t)begins) | ((uintptr_t)state)) & 15)) return HB_BAD_ARGUMENT;
    if (!out || !ends || !decays || !begins || !state || !start || !chunk_row || out_e < e + sums || (sums != 0 && sums != 1)) return HB_BAD_ARGUMENT;
    if (kind == KIND_STATE_SPACE && (!a_log || !dt_bias || !skip || sums)) return HB_BAD_ARGUMENT;
    const int by_four = ((k_stride | q_stride | v_stride | n | e) & 3) == 0 && (((uintptr_t)k | (uintptr_t)q | (uintptr_t)v) & 15) == 0;
    const ChunkArgs a{k, q, v, k_stride, q_stride, v_stride, gate, gate_stride, decay_off, step_off, a_log, dt_bias, skip, ends, (size_t)heads * (e + sums) * n_padded, decays,
                      (__nv_bfloat16*)begins, start, out, out_e, heads, groups, n, n_padded, e, sums, q_scale, by_four, out_e % 2 == 0 && ((uintptr_t)out & 7) == 0};
    if (kind == KIND_STATE_SPACE) return launch_chunks<KIND_STATE_SPACE>(a, chunks, state, slot_stride, state_off, slots, chunk_row, stream);
    if (kind == KIND_GIVEN) return launch_chunks<KIND_GIVEN>(a, chunks, state, slot_stride, state_off, slots, chunk_row, stream);
    return HB_BAD_ARGUMENT;
}
