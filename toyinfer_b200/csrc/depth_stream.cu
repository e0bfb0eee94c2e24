// A float32 residual stream that is averaged over depth after every layer, the norm that reads it, and the token shift.
//
// The stream's history is the embedding X_0 [M, H] and the layers' results X_1, X_2, ..., float32, each a buffer of its own.
// A layer that has n results before it reads y = sum_{j < n} c_j X_j (c: n coefficients; null: y = X_{n-1}) and leaves two
// outputs a and f (engine type, f may be absent) pending:
//     X_n = y + mult * (a + f);      y' = sum_{j < n} d_j X_j + d_n X_n        (d: n + 1 coefficients; null: y' = X_n)
// One kernel does what a layer boundary needs: X_n (written to its buffer), y', and z = y' * rsqrt(mean(y'^2) + eps) * w,
// rounded once into the engine's type.  y itself is never stored: the coefficients that formed it are applied to the same
// loads that form y'.  Without a pending layer y' = y.
//
// Token shift (optional): z'_t = z_t + (z_{t-1} - z_t) * s per channel, formed from the unrounded z and rounded once; z_{t-1}
// is the token before in the SAME sequence.  For a sequence's first token of a step it comes from `prev` (a row per slot or
// per sequence of the step; null: zeros), and a sequence's last z of a step goes to its row of `state`.  A block walks
// `rows_per_block` neighbouring rows with the row before in shared memory; the one before its first row is formed again.
// A caller whose sequences bring several tokens after cached ones must hand in a copy of the state as `prev`: the block
// with a sequence's last row may run before the one with its first.
//
// With `rows` the kernel works on the gathered rows only, without shift, and writes no result (the head's rows).
#include "common.cuh"

namespace {

constexpr int MAX_RESULTS = 256;

struct Results { const float* x[MAX_RESULTS]; };

struct DepthArgs {
    const float* coef_in; const float* coef_out;
    const void* a; const void* f; float mult;
    float* x_out;
    const float* w; float eps;
    void* out; float* sum_out;
    const float* shift; void* shifted;
    const float* prev; int prev_by_slot;
    float* state;
    const int* tok_seq; const int* seq_slot; const int* cu_new;
    const int* rows;
    int n, R, H, M, rows_per_block;
};

template <int V> __device__ __forceinline__ void load_f32(const float* p, float (&x)[V]) {
    if constexpr (V == 4) { const float4 v = *reinterpret_cast<const float4*>(p); x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w; }
    else x[0] = *p;
}
template <int V> __device__ __forceinline__ void store_f32(float* p, const float (&x)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
    else *p = x[0];
}
template <int V> __device__ __forceinline__ void load_t(const float* p, float (&x)[V]) { load_f32<V>(p, x); }
template <int V> __device__ __forceinline__ void store_t(float* p, const float (&x)[V]) { store_f32<V>(p, x); }
template <int V> __device__ __forceinline__ void load_t(const bf16* p, float (&x)[V]) {
    if constexpr (V == 4) {
        struct alignas(8) Four { bf16 v[4]; };
        const Four v = *reinterpret_cast<const Four*>(p);
#pragma unroll
        for (int e = 0; e < 4; e++) x[e] = to_f32(v.v[e]);
    } else x[0] = to_f32(*p);
}
template <int V> __device__ __forceinline__ void store_t(bf16* p, const float (&x)[V]) {
    if constexpr (V == 4) {
        struct alignas(8) Four { bf16 v[4]; } v;
#pragma unroll
        for (int e = 0; e < 4; e++) v.v[e] = from_f32<bf16>(x[e]);
        *reinterpret_cast<Four*>(p) = v;
    } else *p = from_f32<bf16>(x[0]);
}

template <typename T, int V>
__global__ void depth_norm_kernel(const __grid_constant__ Results res, const __grid_constant__ DepthArgs g) {
    ti_pdl_trigger();
    extern __shared__ __align__(16) float sm[];
    const int H = g.H, n = g.n;
    float* cur = sm;                     // [H] the row at hand
    float* before = cur + H;             // [H] the normed row before it (only with a shift)
    float* cin = g.shift ? before + H : before;
    float* cout = cin + n;
    float* red = cout + n + 1;           // [33]
    for (int j = threadIdx.x; j < n; j += blockDim.x) {
        cin[j] = g.coef_in ? g.coef_in[j] : (j == n - 1 ? 1.f : 0.f);
        cout[j] = g.coef_out ? g.coef_out[j] : 0.f;
    }
    if (threadIdx.x == 0) cout[n] = g.coef_out ? g.coef_out[n] : 1.f;
    __syncthreads();
    ti_pdl_sync();
    const T* a = ti_dependent((const T*)g.a);
    const T* f = ti_dependent((const T*)g.f);
    const float* prev = ti_dependent(g.prev);
    T* out = (T*)g.out;
    T* shifted = (T*)g.shifted;

    // y' of row m into cur[]; returns the thread's share of its sum of squares.  own: the row is this block's to write
    auto stream_row = [&](int m, bool ok, bool own, int r) {
        const size_t base = (size_t)m * H;
        float ss = 0.f;
        for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
            float y[V], yn[V];
#pragma unroll
            for (int e = 0; e < V; e++) { y[e] = 0.f; yn[e] = 0.f; }
#pragma unroll 4
            for (int j = 0; j < n; j++) {
                float x[V];
                load_f32<V>(res.x[j] + base + i, x);
                const float ci = cin[j], co = cout[j];
#pragma unroll
                for (int e = 0; e < V; e++) { y[e] = fmaf(ci, x[e], y[e]); yn[e] = fmaf(co, x[e], yn[e]); }
            }
            if (a) {
                float av[V], fv[V];
                load_t<V>(a + base + i, av);
                if (f) {
                    load_t<V>(f + base + i, fv);
#pragma unroll
                    for (int e = 0; e < V; e++) av[e] += fv[e];
                }
                const float co = cout[n];
#pragma unroll
                for (int e = 0; e < V; e++) { av[e] = fmaf(g.mult, av[e], y[e]); y[e] = fmaf(co, av[e], yn[e]); }
                if (own && g.x_out) store_f32<V>(g.x_out + base + i, av);
            }
            if (!ok) {
#pragma unroll
                for (int e = 0; e < V; e++) y[e] = 0.f;
            }
            store_f32<V>(cur + i, y);
            if (own && g.sum_out) store_f32<V>(g.sum_out + (size_t)r * H + i, y);
#pragma unroll
            for (int e = 0; e < V; e++) ss = fmaf(y[e], y[e], ss);
        }
        return ss;
    };

    const int r0 = blockIdx.x * g.rows_per_block, r1 = min(r0 + g.rows_per_block, g.R);
    // the row before the block's first, when that one continues a sequence inside this step
    int r = r0;
    if (g.shift && r0 > 0 && r0 != g.cu_new[g.tok_seq[r0]]) r = r0 - 1;
    for (; r < r1; r++) {
        const bool own = r >= r0;
        int m = g.rows ? g.rows[r] : r;
        const bool ok = m >= 0 && m < g.M;
        if (!ok) m = 0;
        const float ss = block_sum(stream_row(m, ok, own, r), red);
        if (!out) continue;
        const float inv = rsqrtf(ss / (float)H + g.eps);
        bool first = false, last = false;
        const float* prow = nullptr;
        float* srow = nullptr;
        if (g.shift && own) {
            const int seq = g.tok_seq[r];
            first = r == g.cu_new[seq];
            last = r == g.cu_new[seq + 1] - 1;
            if (first && prev) prow = prev + (size_t)(g.prev_by_slot ? g.seq_slot[seq] : seq) * H;
            if (last && g.state) srow = g.state + (size_t)g.seq_slot[seq] * H;
        }
        for (int i = threadIdx.x * V; i < H; i += blockDim.x * V) {
            float y[V], wv[V];
            load_f32<V>(cur + i, y);
            load_f32<V>(g.w + i, wv);
#pragma unroll
            for (int e = 0; e < V; e++) y[e] = y[e] * inv * wv[e];
            if (own) store_t<V>(out + (size_t)r * H + i, y);
            if (g.shift) {
                if (own) {
                    float p[V], s[V];
                    if (!first) load_f32<V>(before + i, p);
                    else if (prow) load_f32<V>(prow + i, p);
                    else {
#pragma unroll
                        for (int e = 0; e < V; e++) p[e] = 0.f;
                    }
                    load_f32<V>(g.shift + i, s);
#pragma unroll
                    for (int e = 0; e < V; e++) s[e] = fmaf(p[e] - y[e], s[e], y[e]);
                    store_t<V>(shifted + (size_t)r * H + i, s);
                    if (srow) store_f32<V>(srow + i, y);
                }
                store_f32<V>(before + i, y);
            }
        }
    }
}

inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

// results: n pointers to float32 [M, H]; coef_in: float32 [n] or null; coef_out: float32 [n + 1] or null; a, f: [M, H] of the
// engine's type or null (f needs a); x_out: float32 [M, H] (may be null); w: float32 [H]; out: [R, H] of the engine's type or
// null; sum_out: float32 [R, H] or null (y' itself).  shift: float32 [H] or null, with shifted [R, H] of the engine's type,
// prev (float32 rows of H, by slot or by sequence) or null, state (float32 rows of H by slot) or null, and the step's tok_seq,
// seq_slot and cu_new.  rows: null (every row, R == M) or R row indices (then no shift and no x_out).
extern "C" int ti_depth_norm(const void* const* results, int n, const float* coef_in, const float* coef_out, const void* a,
                             const void* f, float mult, float* x_out, const float* w, float eps, void* out, float* sum_out,
                             const float* shift, void* shifted, const float* prev, int prev_by_slot, float* state,
                             const int* tok_seq, const int* seq_slot, const int* cu_new, const int* rows, int R, int H, int M,
                             int one_token_each, int dtype, cudaStream_t stream) {
    if (R == 0) return 0;
    TI_REQUIRE(R > 0 && H > 0 && M > 0 && n >= 1, "depth_norm: bad sizes R=%d H=%d M=%d results=%d", R, H, M, n);
    TI_REQUIRE(n <= MAX_RESULTS, "depth_norm: a history of %d results is not supported (up to %d)", n, MAX_RESULTS);
    TI_REQUIRE(rows || R == M, "depth_norm: without row indices every row is taken (R=%d, M=%d)", R, M);
    TI_REQUIRE(!rows || (!shift && !x_out), "depth_norm: gathered rows take no shift and write no result");
    TI_REQUIRE(a || (!f && !x_out), "depth_norm: a second output or a result without a first output");
    TI_REQUIRE(!shift || (shifted && tok_seq && seq_slot && cu_new && out), "depth_norm: the shift needs its output and the step's sequences");
    TI_REQUIRE(!out || w, "depth_norm: the norm needs its weight");
    Results res = {};
    bool vec = (H & 3) == 0 && al16(a) && al16(f) && al16(x_out) && al16(w) && al16(out) && al16(sum_out) && al16(shift) &&
               al16(shifted) && al16(prev) && al16(state);
    for (int j = 0; j < n; j++) {
        TI_REQUIRE(results[j], "depth_norm: result %d is missing", j);
        res.x[j] = (const float*)results[j];
        vec = vec && al16(results[j]);
    }
    const size_t smem = ((size_t)H * (shift ? 2 : 1) + 2 * n + 1 + 33) * sizeof(float);
    TI_REQUIRE(smem <= 200 * 1024, "depth_norm: rows of %d elements do not fit shared memory", H);
    // Rows per block and threads, measured at a width of 2,048 with 3 and 12 results: few rows want a row's channels over many
    // threads, many rows fewer rows that are formed twice (2,048 rows, 3 results: 31.9 us at 3 rows and 256 threads, 27.4 at 4
    // and 512; 8,192 rows: 99 us at one row, 80.6 at 8 and 256; 512 rows: 13.9 us at 256 threads, 10.7 at 512).
    int per = 1;
    if (shift && !one_token_each) per = R <= 1024 ? 1 : R < 2048 ? 2 : R <= 4096 ? 4 : 8;
    DepthArgs g{coef_in, coef_out, a, f, mult, x_out, w, eps, out, sum_out, shift, shifted, prev, prev_by_slot, state, tok_seq, seq_slot,
                cu_new, rows, n, R, H, M, per};
    const int lanes = vec ? (H + 3) / 4 : H;
    const int cap = R <= 296 ? 1024 : R <= 1024 || (R >= 2048 && R <= 4096) ? 512 : 256;
    int threads = (lanes + 31) / 32 * 32;
    threads = threads > cap ? cap : threads;
    return ti_dispatch_dtype(dtype, [&](auto t) -> int {
        using T = decltype(t);
        auto go = [&](auto kernel) -> int {
            if (smem > 48 * 1024) TI_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            TI_CUDA(ti_launch_class<1>(kernel, dim3((R + per - 1) / per), dim3(threads), smem, stream, res, g));
            TI_CHECK_LAUNCH("depth_norm");
            return 0;
        };
        return vec ? go(depth_norm_kernel<T, 4>) : go(depth_norm_kernel<T, 1>);
    });
}
