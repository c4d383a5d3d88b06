// What stands between a part's output and the next part's input where the norm computes no statistics, entry by entry:
//
//   v = x[r] + (delta[r] + delta_b) * sigmoid(gate[r] + gate_b)      each of the three but delta may be missing, and delta too
//   history[terms - 1][r] = v;   v <- sum_{j < terms} c[j] * history[j][r]                  (terms > 0: a sum over the depth)
//   x[r] = v                                                                            when the stream changed and rows is null
//   y[i] = tanh(alpha v) * w + b,  or v itself without w                                                  one rounding to T
//
// with row r = rows ? rows[i] : i.  Everything is float; x and history are float.  With rows nothing but y is written.
// The embedding with learned positions is the same kind of kernel:  x[i] = N(table[tok_i] * scale + positions[pos_i]).
//
// A thread takes eight neighbouring entries with 16-byte accesses where the layout allows it, else one; the grid covers
// the entries of all rows, so that few rows still fill the GPU.
#include "common.cuh"

struct StreamStepArgs {
    float* x;
    const void* delta;
    const float* delta_b;
    const void* gate;
    const float* gate_b;
    float* history;
    const float* c;
    const int* rows;
    const float* alpha;
    const float* w;
    const float* b;
    void* y;
    long long hstride;
    int ldg, terms, n_out, d;
};

template <int V> __device__ __forceinline__ void ss_loadf(const float* p, float (&f)[V]) {
    if constexpr (V == 8) load8(p, f);
    else f[0] = *p;
}
template <typename T, int V> __device__ __forceinline__ void ss_load(const T* p, float (&f)[V]) {
    if constexpr (V == 8) load8(p, f);
    else f[0] = ldf(p);
}
template <typename T, int V> __device__ __forceinline__ void ss_store(T* p, const float (&f)[V]) {
    if constexpr (V == 8) store8(p, f);
    else stf(p, f[0]);
}

template <typename T, int V>
__global__ void __launch_bounds__(128) stream_step_kernel(const StreamStepArgs a) {
    const int per_row = a.d / V;
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const bool mine = idx < (long long)a.n_out * per_row;
    const int i = mine ? (int)(idx / per_row) : 0, col = mine ? (int)(idx - (long long)i * per_row) * V : 0;
    // weights: nothing of the step writes them
    float w[V], b[V], gb[V], db[V];
#pragma unroll
    for (int e = 0; e < V; ++e) w[e] = b[e] = gb[e] = db[e] = 0.f;
    if (a.w) {
        ss_loadf<V>(a.w + col, w);
        ss_loadf<V>(a.b + col, b);
    }
    if (a.gate_b) ss_loadf<V>(a.gate_b + col, gb);
    if (a.delta_b) ss_loadf<V>(a.delta_b + col, db);
    const float alpha = a.alpha ? *a.alpha : 0.f;
    pdl_sync();
    if (!mine) return;
    const int r = a.rows ? a.rows[i] : i;
    const size_t at = (size_t)r * a.d + col;
    float v[V];
    ss_loadf<V>(a.x + at, v);
    if (a.delta) {
        float u[V];
        ss_load<T, V>(static_cast<const T*>(a.delta) + at, u);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] += db[e];
        if (a.gate) {
            float g[V];
            ss_load<T, V>(static_cast<const T*>(a.gate) + (size_t)r * a.ldg + col, g);
#pragma unroll
            for (int e = 0; e < V; ++e) u[e] *= 1.0f / (1.0f + expf(-(g[e] + gb[e])));
        }
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] += u[e];
    }
    if (a.terms > 0) {
        const int last = a.terms - 1;
        if (!a.rows) ss_store<float, V>(a.history + (size_t)last * a.hstride + at, v);
        float s[V];
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] = 0.f;
        const float* hp = a.history + at;
#pragma unroll 4
        for (int j = 0; j < last; ++j, hp += a.hstride) {
            float h[V];
            ss_loadf<V>(hp, h);
            const float cj = a.c[j];
#pragma unroll
            for (int e = 0; e < V; ++e) s[e] += cj * h[e];
        }
        const float cl = a.c[last];
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = s[e] + cl * v[e];
    }
    if (!a.rows && (a.delta || a.terms > 0)) ss_store<float, V>(a.x + at, v);
    if (a.y) {
        if (a.w) {
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = tanhf(alpha * v[e]) * w[e] + b[e];
        }
        ss_store<T, V>(static_cast<T*>(a.y) + (size_t)i * a.d + col, v);
    }
}

template <typename T>
static int stream_step_launch(const StreamStepArgs& a, cudaStream_t s) {
    if (a.n_out < 0 || a.d <= 0 || a.terms < 0) return TB_ERR_ARG;
    if (a.n_out == 0) return 0;
    if (!a.x) return TB_ERR_ARG;
    if (a.terms > 0 && (!a.history || !a.c || a.hstride < a.d)) return TB_ERR_ARG;
    if ((a.gate || a.delta_b) && !a.delta) return TB_ERR_ARG;
    if (a.gate ? a.ldg < a.d : a.gate_b != nullptr) return TB_ERR_ARG;
    if ((a.w != nullptr) != (a.alpha != nullptr) || (a.w != nullptr) != (a.b != nullptr)) return TB_ERR_ARG;
    if (a.rows && !a.y) return TB_ERR_ARG;
    const uintptr_t all = (uintptr_t)a.x | (uintptr_t)a.delta | (uintptr_t)a.delta_b | (uintptr_t)a.gate | (uintptr_t)a.gate_b |
                          (uintptr_t)a.history | (uintptr_t)a.w | (uintptr_t)a.b | (uintptr_t)a.y;
    const bool vec = a.d % 8 == 0 && a.ldg % 8 == 0 && a.hstride % 4 == 0 && (all & 15) == 0;
    const long long n = (long long)a.n_out * (a.d / (vec ? 8 : 1));
    const int threads = n >= 128 * 148 ? 128 : 32;      // few rows: small blocks, so that every SM has some
    const long long blocks = (n + threads - 1) / threads;
    if (blocks > 0x7fffffffll) return TB_ERR_UNSUPPORTED;
    if (vec) TB_LAUNCH((stream_step_kernel<T, 8>), (unsigned)blocks, threads, 0, s, a);
    else TB_LAUNCH((stream_step_kernel<T, 1>), (unsigned)blocks, threads, 0, s, a);
    return tb_last_error();
}

// ---- the embedding with learned positions --------------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(128)
embed_learned_kernel(const int* __restrict__ tokens, const int* __restrict__ positions, const T* __restrict__ table,
                     const T* __restrict__ ptable, float* __restrict__ x, int nt, int d, float scale,
                     const float* __restrict__ alpha, const float* __restrict__ w, const float* __restrict__ b) {
    pdl_sync();
    const int per_row = d / V;
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)nt * per_row) return;
    const int i = (int)(idx / per_row), col = (int)(idx - (long long)i * per_row) * V;
    float e0[V], p0[V];
    ss_load<T, V>(table + (size_t)tokens[i] * d + col, e0);
    ss_load<T, V>(ptable + (size_t)positions[i] * d + col, p0);
#pragma unroll
    for (int e = 0; e < V; ++e) e0[e] = e0[e] * scale + p0[e];
    if (w) {
        const float al = *alpha;
        float wv[V], bv[V];
        ss_loadf<V>(w + col, wv);
        ss_loadf<V>(b + col, bv);
#pragma unroll
        for (int e = 0; e < V; ++e) e0[e] = tanhf(al * e0[e]) * wv[e] + bv[e];
    }
    ss_store<float, V>(x + (size_t)i * d + col, e0);
}

template <typename T>
static int embed_learned_launch(const int* tokens, const int* positions, const void* table, const void* ptable, float* x,
                                int nt, int d, float scale, const float* alpha, const float* w, const float* b,
                                cudaStream_t s) {
    if (nt == 0) return 0;
    if (nt < 0 || d <= 0 || !tokens || !positions || !table || !ptable || !x) return TB_ERR_ARG;
    if ((w != nullptr) != (alpha != nullptr) || (w != nullptr) != (b != nullptr)) return TB_ERR_ARG;
    const bool vec = d % 8 == 0 &&
                     (((uintptr_t)table | (uintptr_t)ptable | (uintptr_t)x | (uintptr_t)w | (uintptr_t)b) & 15) == 0;
    const long long n = (long long)nt * (d / (vec ? 8 : 1)), blocks = (n + 127) / 128;
    if (blocks > 0x7fffffffll) return TB_ERR_UNSUPPORTED;
    if (vec)
        TB_LAUNCH((embed_learned_kernel<T, 8>), (unsigned)blocks, 128, 0, s, tokens, positions, (const T*)table,
                  (const T*)ptable, x, nt, d, scale, alpha, w, b);
    else
        TB_LAUNCH((embed_learned_kernel<T, 1>), (unsigned)blocks, 128, 0, s, tokens, positions, (const T*)table,
                  (const T*)ptable, x, nt, d, scale, alpha, w, b);
    return tb_last_error();
}

extern "C" {
#define TB_STREAM_STEP(SFX, T)                                                                                        \
    int tb_stream_step_##SFX(float* x, const void* delta, const float* delta_b, const void* gate, int ldg,            \
                             const float* gate_b, float* history, long long hstride, const float* c, int terms,       \
                             const int* rows, const float* alpha, const float* w, const float* b, void* y, int n_out, \
                             int d, cudaStream_t s) {                                                                 \
        return stream_step_launch<T>(StreamStepArgs{x, delta, delta_b, gate, gate_b, history, c, rows, alpha, w, b,   \
                                                    y, hstride, ldg, terms, n_out, d}, s);                            \
    }                                                                                                                 \
    int tb_embed_learned_##SFX(const int* tokens, const int* positions, const void* table, const void* ptable,        \
                               float* x, int nt, int d, float scale, const float* alpha, const float* w,              \
                               const float* b, cudaStream_t s) {                                                      \
        return embed_learned_launch<T>(tokens, positions, table, ptable, x, nt, d, scale, alpha, w, b, s);            \
    }
TB_STREAM_STEP(f32, float)
TB_STREAM_STEP(bf16, __nv_bfloat16)
}

#include "tape.h"
TB_TAPE_REGISTER(tb_stream_step_f32)
TB_TAPE_REGISTER(tb_stream_step_bf16)
TB_TAPE_REGISTER(tb_embed_learned_f32)
TB_TAPE_REGISTER(tb_embed_learned_bf16)
