// A linear attention whose memory fades per key channel, state in float.
//
// Per head, with a state S [dim, vdim] that is zero when a sequence starts (rows: key channels):
//
//   S <- diag(alpha_t) S + k_t v_t^T;    o_t = S^T q_t;      alpha = sigmoid(z)^(1 / tau),  z = A2 (A1 x) + bias
//
// State of one slot (floats): S [H][dim][vdim].
//
//   gated_linear_prep_kernel   prompts: one float record per (token, head) for the scan of decay_memory.cu, whose output
//                              is read before the token is written: o_t = S_{t-1}^T (alpha q) + (q . k) v
//   gated_linear_step_kernel   one token per sequence: decays, the state's way through the registers, the head's norm and
//                              the gate in one kernel; a block = a sequence x a head
// Everything that enters the recurrence is float on both paths; q, k, v and the gate have the activations' type.
#include "memory_common.cuh"

__device__ __forceinline__ float gl_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// sigmoid(z)^(1 / tau)
__device__ __forceinline__ float gl_decay(float z, float inv_tau) { return expf(-gl_softplus(-z) * inv_tau); }

struct GatedLinearArgs {
    const void* z;          // [nt, ldz]: q (H dim) | k (H dim) | v (H vdim) | gate (H vdim)
    const float* pre;       // [nt, H dim]  A2 (A1 x)
    const float* bias;      // [H dim]
    float* rec;             // [H, nt, record]: alpha q | k | alpha (dm_rows(dim) each) | v (vp) | q . k, 0, 0, 0
    int nt, ldz, H, dim, vdim, vp;
    float inv_tau, qscale;
};

// A warp per (token, head); VEC: four neighbouring entries a lane and access.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) gated_linear_prep_kernel(const GatedLinearArgs p) {
    pdl_sync();
    constexpr int V = VEC ? 4 : 1;
    const int lane = threadIdx.x & 31;
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (row >= p.nt * p.H) return;
    const int t = row / p.H, h = row - t * p.H, dim = p.dim, vdim = p.vdim, hk = p.H * dim;
    const int DP = dm_rows(dim);
    float* rec = p.rec + ((size_t)h * p.nt + t) * (3 * DP + p.vp + 4);
    const T* z = static_cast<const T*>(p.z) + (size_t)t * p.ldz;
    float dot = 0.f;
    for (int c = lane * V; c < DP; c += 32 * V) {
        float q[V], k[V], w[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            q[e] = k[e] = 0.f;
            w[e] = 1.f;
        }
        if (c < dim) {
            float pre[V], b[V];
            dm_load<T, V>(z + h * dim + c, q);
            dm_load<T, V>(z + hk + h * dim + c, k);
            dm_load<float, V>(p.pre + (size_t)t * hk + h * dim + c, pre);
            dm_load<float, V>(p.bias + h * dim + c, b);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                w[e] = gl_decay(pre[e] + b[e], p.inv_tau);
                q[e] *= p.qscale;
                dot += q[e] * k[e];
                q[e] *= w[e];
            }
        }
        dm_store<V>(rec + c, q);
        dm_store<V>(rec + DP + c, k);
        dm_store<V>(rec + 2 * DP + c, w);
    }
    for (int c = lane * V; c < p.vp; c += 32 * V) {
        float v[V];
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = 0.f;
        if (c < vdim) dm_load<T, V>(z + 2 * hk + h * vdim + c, v);
        dm_store<V>(rec + 3 * DP + c, v);
    }
    dot = warp_sum(dot);
    if (lane < 4) rec[3 * DP + p.vp + lane] = lane == 0 ? dot : 0.f;
}

template <typename T>
static int gated_linear_prep_launch(const GatedLinearArgs& p, cudaStream_t s) {
    if (p.nt < 0 || p.H <= 0 || p.dim <= 0 || p.vdim <= 0 || p.vp < p.vdim || p.vp % 4 || p.ldz < 2 * p.H * (p.dim + p.vdim))
        return TB_ERR_ARG;
    if (p.dim > 256) return TB_ERR_UNSUPPORTED;
    if (p.nt == 0) return 0;
    const bool vec = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.ldz % 4 == 0 &&
                     (((uintptr_t)p.z | (uintptr_t)p.pre | (uintptr_t)p.bias) & 15) == 0;
    const int grid = (int)(((long long)p.nt * p.H + 7) / 8);
    if (vec) TB_LAUNCH((gated_linear_prep_kernel<T, true>), grid, 256, 0, s, p);
    else TB_LAUNCH((gated_linear_prep_kernel<T, false>), grid, 256, 0, s, p);
    return tb_last_error();
}

// ---- one token per sequence -------------------------------------------------------------------------------------
struct GatedLinearStepArgs {
    const void* z;          // [nt, ldz]: q | k | v | gate
    const float* a;         // [nt, lda]  A1 x
    const void* a2;         // [H dim, rank]
    const float* bias;      // [H dim]
    const float* norm;      // [H vdim]
    float* state;
    void* y;                // [nt, ldy]
    const int* seq_start;
    const int* slots;
    long long pitch;
    int nt, ldz, lda, ldy, H, dim, vdim, rank;
    float inv_tau, qscale, eps;
};

// VEC: four columns a thread and access (vdim a multiple of four), else one.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) gated_linear_step_kernel(const GatedLinearStepArgs p) {
    constexpr int V = VEC ? 4 : 1;
    constexpr int U = 8;                    // rows asked for together
    extern __shared__ __align__(16) float gl_sm[];
    const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int dim = p.dim, vdim = p.vdim, hk = p.H * dim, hv = p.H * vdim;
    const int rank4 = (p.rank + 3) / 4 * 4, dim4 = (dim + 3) / 4 * 4, vdim4 = (vdim + 3) / 4 * 4;
    const int nc = vdim / V, G = 256 / nc;  // columns' threads, groups of rows
    float* ta = gl_sm;                      // [rank4]
    float* q_s = ta + rank4;                // [dim4] each
    float* k_s = q_s + dim4;
    float* w_s = k_s + dim4;
    float* v_s = w_s + dim4;                // [vdim4]
    float* o_s = v_s + vdim4;               // [G][vdim4]
    __shared__ float red[33];
    const float nw = tid < vdim ? p.norm[h * vdim + tid] : 0.f;      // weights: nothing of the step writes them
    pdl_sync();
    const int t = p.seq_start[b];
    float* S = p.state + (size_t)p.slots[b] * p.pitch + (size_t)h * dim * vdim;
    const T* z = static_cast<const T*>(p.z) + (size_t)t * p.ldz;
    // the state's first rows are on their way while the decays are made
    const int rg = tid / nc, c = (tid - rg * nc) * V;
    float s[U][V];
    auto fetch = [&](int r0) {
#pragma unroll
        for (int q = 0; q < U; ++q) {
            const int r = r0 + q * G;
            if (r < dim) dm_load<float, V>(S + (size_t)r * vdim + c, s[q]);
        }
    };
    if (rg < G) fetch(rg);
    for (int q = tid; q < p.rank; q += 256) ta[q] = p.a[(size_t)t * p.lda + q];
    if (tid < dim) {
        q_s[tid] = ldf(z + h * dim + tid) * p.qscale;
        k_s[tid] = ldf(z + hk + h * dim + tid);
    }
    float gate = 0.f;
    if (tid < vdim) {
        v_s[tid] = ldf(z + 2 * hk + h * vdim + tid);
        gate = ldf(z + 2 * hk + hv + h * vdim + tid);
    }
    __syncthreads();
    {
        // adjacent lanes share a channel's row of A2
        const int parts = 256 / dm_rows(dim), ch = tid / parts, part = tid - ch * parts;
        float acc = 0.f;
        if (ch < dim)
            acc = decay_dot<T>(static_cast<const T*>(p.a2) + (size_t)(h * dim + ch) * p.rank, ta, p.rank, part, parts);
        for (int o = parts >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (ch < dim && part == 0) w_s[ch] = gl_decay(acc + p.bias[h * dim + ch], p.inv_tau);
    }
    __syncthreads();
    if (rg < G) {
        float acc[V], v[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            acc[e] = 0.f;
            v[e] = v_s[c + e];
        }
        for (int r0 = rg; r0 < dim; r0 += G * U) {
            if (r0 != rg) fetch(r0);
#pragma unroll
            for (int q = 0; q < U; ++q) {
                const int r = r0 + q * G;
                if (r >= dim) break;
                const float qq = q_s[r], kk = k_s[r], ww = w_s[r];
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    s[q][e] = s[q][e] * ww + kk * v[e];
                    acc[e] += s[q][e] * qq;
                }
                dm_store<V>(S + (size_t)r * vdim + c, s[q]);
            }
        }
#pragma unroll
        for (int e = 0; e < V; ++e) o_s[rg * vdim4 + c + e] = acc[e];
    }
    __syncthreads();
    float o = 0.f;
    if (tid < vdim)
        for (int g = 0; g < G; ++g) o += o_s[g * vdim4 + tid];
    const float rs = 1.0f / sqrtf(block_sum(o * o, red) / (float)vdim + p.eps);
    if (tid < vdim)
        stf(static_cast<T*>(p.y) + (size_t)t * p.ldy + h * vdim + tid, o * rs * nw * (gate / (1.0f + expf(-gate))));
}

template <typename T>
static int gated_linear_step_launch(const GatedLinearStepArgs& p, int B, cudaStream_t s) {
    if (B < 0 || p.nt < B || p.H <= 0 || p.dim <= 0 || p.vdim <= 0 || p.rank <= 0 || p.lda < p.rank ||
        p.ldy < p.H * p.vdim || p.ldz < 2 * p.H * (p.dim + p.vdim) || p.pitch < (long long)p.H * p.dim * p.vdim)
        return TB_ERR_ARG;
    if (p.dim > 256 || p.vdim > 256 || p.rank > 4096 || (p.rank % 8 == 0 && ((uintptr_t)p.a2 & 15))) return TB_ERR_UNSUPPORTED;
    if (B == 0) return 0;
    const bool vec = p.vdim % 4 == 0 && p.pitch % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
    const int dim4 = (p.dim + 3) / 4 * 4, vdim4 = (p.vdim + 3) / 4 * 4, G = 256 / (p.vdim / (vec ? 4 : 1));
    const size_t smem = ((size_t)(p.rank + 3) / 4 * 4 + 3 * (size_t)dim4 + (size_t)(1 + G) * vdim4) * sizeof(float);
    if (smem > 48 * 1024) return TB_ERR_UNSUPPORTED;
    if (vec) TB_LAUNCH((gated_linear_step_kernel<T, true>), dim3(B, p.H), 256, smem, s, p);
    else TB_LAUNCH((gated_linear_step_kernel<T, false>), dim3(B, p.H), 256, smem, s, p);
    return tb_last_error();
}

extern "C" {
// vp: floats of a record's values (tb_decay_scan_rect_record_size less the three vectors and the last four floats).
#define TB_GATED_LINEAR(SFX, T)                                                                                       \
    int tb_gated_linear_prep_##SFX(const void* z, int ldz, const float* pre, const float* bias, float* rec, int nt,   \
                                   int H, int dim, int vdim, int record, float inv_tau, float qscale,                 \
                                   cudaStream_t s) {                                                                  \
        if ((uintptr_t)rec & 15) return TB_ERR_ARG;                                                                   \
        return gated_linear_prep_launch<T>(GatedLinearArgs{z, pre, bias, rec, nt, ldz, H, dim, vdim,                  \
                                                           record - 3 * dm_rows(dim) - 4, inv_tau, qscale}, s);       \
    }                                                                                                                 \
    int tb_gated_linear_step_##SFX(const void* z, int ldz, const float* a, int lda, const void* a2,                   \
                                   const float* bias, const float* norm, float* state, long long pitch, void* y,      \
                                   int ldy, const int* seq_start, const int* slots, int nt, int B, int H, int dim,    \
                                   int vdim, int rank, float inv_tau, float qscale, float eps, cudaStream_t s) {      \
        return gated_linear_step_launch<T>(GatedLinearStepArgs{z, a, a2, bias, norm, state, y, seq_start, slots,      \
                                                               pitch, nt, ldz, lda, ldy, H, dim, vdim, rank, inv_tau, \
                                                               qscale, eps}, B, s);                                   \
    }
TB_GATED_LINEAR(f32, float)
TB_GATED_LINEAR(bf16, __nv_bfloat16)
}

#include "tape.h"
TB_TAPE_REGISTER(tb_gated_linear_prep_f32)
TB_TAPE_REGISTER(tb_gated_linear_prep_bf16)
TB_TAPE_REGISTER(tb_gated_linear_step_f32)
TB_TAPE_REGISTER(tb_gated_linear_step_bf16)
