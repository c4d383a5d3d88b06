// A delta rule in which what fades, what is removed and what is written are three different things, state in float.
//
// Per head, with a state S [dim, dim] that is zero when a sequence starts (rows: key channels, columns: values) and the
// unit key u = k / sqrt(sum k^2 + 1e-6):
//
//   S_t = diag(w) S - (a u) (u^T S) + k v^T     both terms read the old S;      o_t = S_t^T r
//   w = exp(-e^(-1/2) sigmoid(W2 tanh(x1) + w0))   the decay, per head and key channel
//   a = sigmoid(x2 + b)                            the removal rate, per head and key channel
//
// State of one slot (floats): S [H][dim][dim].
//
// The key is its length times u, so with v' = |k| v and the sums over the old state p_j = u . S[:, j]:
//   o_j = (w r) . S[:, j] - (r . a u) p_j + (r . u) v'_j;      S[i][j] <- w_i S[i][j] - (a u)_i p_j + u_i v'_j
//
//   split_delta_prep_kernel   prompts: one float record per (token, head), w r | u | w | -a u | v' | -(r . a u), r . u, 0, 0,
//                             those of a head one behind the other
//   split_delta_scan_kernel   prompts: the recurrence token by token, a block = a sequence x a head x some columns of S, whose
//                             rows are split over adjacent lanes, in registers; the lanes meet once a token for p, and
//                             for the outputs only once a stage of several tokens
//   split_delta_step_kernel   one token per sequence: a block = a sequence x a head; everything between the projections and
//                             the output product in one kernel, the head's state in registers between the two passes
// Everything that enters the recurrence is float on both paths; r, k, v and the gate have the activations' type.
#include "memory_common.cuh"
#include "tc_common.cuh"                // bulk copies, barriers with bounded waits

#define SD_UNIT_EPS 1e-6f
#define SD_RATE 0.60653065971263342f    // e^(-1/2)

constexpr int SD_STEP = 512;            // threads of a step block

__host__ __device__ inline int sd_record(int dim) { return 5 * dm_rows(dim) + 4; }
__device__ __forceinline__ float sd_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float sd_decay(float z) { return expf(-SD_RATE * sd_sigmoid(z)); }

struct SplitDeltaArgs {
    const void* z;          // [nt, ldz]: r | k | v | gate, H dim each
    const float* az;        // [nt, lda]  pre-activation of the removal rate
    const float* ba;        // [H dim]
    const float* pre;       // [nt, H dim]  W2 tanh(.)
    const float* w0;        // [H dim]
    float* rec;             // [H, nt, sd_record]
    int nt, ldz, lda, H, dim;
};

// A warp per (token, head), NCH pieces of V neighbouring entries a lane (dm_rows(dim) <= 32 V NCH).
template <typename T, int V, int NCH>
__global__ void __launch_bounds__(256) split_delta_prep_kernel(const SplitDeltaArgs p) {
    pdl_sync();
    const int lane = threadIdx.x & 31;
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (row >= p.nt * p.H) return;
    const int t = row / p.H, h = row - t * p.H, dim = p.dim, hd = p.H * dim;
    const int DP = dm_rows(dim);
    float* rec = p.rec + ((size_t)h * p.nt + t) * sd_record(dim);
    const T* z = static_cast<const T*>(p.z) + (size_t)t * p.ldz + h * dim;
    float k[NCH][V], ss = 0.f;
#pragma unroll
    for (int j = 0; j < NCH; ++j) {
        const int c = (lane + 32 * j) * V;
#pragma unroll
        for (int e = 0; e < V; ++e) k[j][e] = 0.f;
        if (c < dim) dm_load<T, V>(z + hd + c, k[j]);
#pragma unroll
        for (int e = 0; e < V; ++e) ss += k[j][e] * k[j][e];
    }
    const float len = sqrtf(warp_sum(ss) + SD_UNIT_EPS), inv = 1.0f / len;
    float rau = 0.f, ru = 0.f;
#pragma unroll
    for (int j = 0; j < NCH; ++j) {
        const int c = (lane + 32 * j) * V;
        if (c >= DP) break;
        float rw[V], u[V], w[V], na[V], v[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            rw[e] = u[e] = na[e] = v[e] = 0.f;
            w[e] = 1.f;
        }
        if (c < dim) {
            float r[V], az[V], ba[V], pre[V], w0[V];
            dm_load<T, V>(z + c, r);
            dm_load<T, V>(z + 2 * hd + c, v);
            dm_load<float, V>(p.az + (size_t)t * p.lda + h * dim + c, az);
            dm_load<float, V>(p.ba + h * dim + c, ba);
            dm_load<float, V>(p.pre + (size_t)t * hd + h * dim + c, pre);
            dm_load<float, V>(p.w0 + h * dim + c, w0);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                u[e] = k[j][e] * inv;
                w[e] = sd_decay(pre[e] + w0[e]);
                na[e] = -sd_sigmoid(az[e] + ba[e]) * u[e];
                rw[e] = r[e] * w[e];
                v[e] *= len;
                rau += r[e] * na[e];
                ru += r[e] * u[e];
            }
        }
        dm_store<V>(rec + c, rw);
        dm_store<V>(rec + DP + c, u);
        dm_store<V>(rec + 2 * DP + c, w);
        dm_store<V>(rec + 3 * DP + c, na);
        dm_store<V>(rec + 4 * DP + c, v);
    }
    rau = warp_sum(rau);
    ru = warp_sum(ru);
    if (lane < 4) rec[5 * DP + lane] = lane == 0 ? rau : lane == 1 ? ru : 0.f;
}

template <typename T>
static int split_delta_prep_launch(const SplitDeltaArgs& p, cudaStream_t s) {
    if (p.nt < 0 || p.H <= 0 || p.dim <= 0 || p.ldz < 4 * p.H * p.dim || p.lda < p.H * p.dim) return TB_ERR_ARG;
    if (p.dim > 256) return TB_ERR_UNSUPPORTED;
    if (p.nt == 0) return 0;
    const bool vec = p.dim % 4 == 0 && p.ldz % 4 == 0 && p.lda % 4 == 0 &&
                     (((uintptr_t)p.z | (uintptr_t)p.az | (uintptr_t)p.ba | (uintptr_t)p.pre | (uintptr_t)p.w0) & 15) == 0;
    const int grid = (int)(((long long)p.nt * p.H + 7) / 8);
    if (vec && p.dim <= 128) TB_LAUNCH((split_delta_prep_kernel<T, 4, 1>), grid, 256, 0, s, p);
    else if (vec) TB_LAUNCH((split_delta_prep_kernel<T, 4, 2>), grid, 256, 0, s, p);
    else TB_LAUNCH((split_delta_prep_kernel<T, 1, 8>), grid, 256, 0, s, p);
    return tb_last_error();
}

// ---- the scan ------------------------------------------------------------------------------------------------
struct SplitDeltaScanArgs {
    const float* rec;
    float* state;           // [slots, pitch]
    int* error;             // set by a wait that runs out
    float* out;             // [nt, H dim]
    const int* seq_start;
    const int* slots;
    long long pitch;
    int nt, H, dim;
};

// RPT rows of C columns per thread, SPLIT lanes per column (SPLIT * RPT = dm_rows(dim)): THREADS / SPLIT * C columns a
// block.  The records of TOK tokens at a time are one bulk copy to shared memory, STAGES - 1 stages ahead.
template <int RPT, int SPLIT, int C, int THREADS, int TOK, int STAGES>
__global__ void __launch_bounds__(THREADS) split_delta_scan_kernel(const SplitDeltaScanArgs a) {
    pdl_sync();
    constexpr int DP = RPT * SPLIT;
    constexpr int COLS = THREADS / SPLIT * C;
    constexpr int ROW = 5 * DP + 4;                     // a record
    constexpr int NV = TOK * C;
    static_assert(NV % SPLIT == 0, "every lane ends with as many sums");
    extern __shared__ __align__(16) float sd_sm[];      // [STAGES][TOK][ROW]
    __shared__ __align__(8) unsigned long long bars[STAGES];
    const int b = blockIdx.x, h = blockIdx.y;
    const int tid = threadIdx.x, part = tid & (SPLIT - 1), cl = tid / SPLIT * C;
    const int col = blockIdx.z * COLS + cl;
    const int dim = a.dim, H = a.H;
    const int t0 = a.seq_start[b], t1 = a.seq_start[b + 1];
    if (t0 >= t1) return;
    float* S = a.state + (size_t)a.slots[b] * a.pitch + (size_t)h * dim * dim;
    F2 s[C][RPT / 2];                                   // rows 2i, 2i + 1 of this lane's
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
        for (int i = 0; i < RPT / 2; ++i) {
            const int r = ((i >> 1) * SPLIT + part) * 4 + (i & 1) * 2;
            s[c][i].f.x = (r < dim && col + c < dim) ? S[(size_t)r * dim + col + c] : 0.f;
            s[c][i].f.y = (r + 1 < dim && col + c < dim) ? S[(size_t)(r + 1) * dim + col + c] : 0.f;
        }
    const float* rec = a.rec + (size_t)h * a.nt * ROW;
    const uint32_t bar0 = smem_u32(bars);
    if (tid == 0) {
        for (int q = 0; q < STAGES; ++q) mbar_init(bar0 + 8u * q, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    const int stages = (t1 - t0 + TOK - 1) / TOK;
    auto issue = [&](int q) {
        const int ts = t0 + q * TOK, n = min(TOK, t1 - ts);
        float* to = sd_sm + (size_t)(q % STAGES) * (TOK * ROW);
        if (tid == 0) {
            const uint32_t bytes = (uint32_t)(n * ROW) * sizeof(float);
            mbar_expect_tx(bar0 + 8u * (q % STAGES), bytes);
            bulk_load(smem_u32(to), rec + (size_t)ts * ROW, bytes, bar0 + 8u * (q % STAGES));
        }
        // tokens behind the last: nothing is written, nothing fades, nothing is read (so that a stage has no branches)
        for (int idx = n * ROW + tid; idx < TOK * ROW; idx += THREADS) {
            const int e = idx % ROW;
            to[idx] = e >= 2 * DP && e < 3 * DP ? 1.f : 0.f;
        }
    };
    int issued = 0;
    for (; issued < STAGES - 1 && issued < stages; ++issued) issue(issued);
    for (int st = 0; st < stages; ++st) {
        const bool ok = mbar_wait(bar0 + 8u * (st % STAGES), (st / STAGES) & 1, a.error, 33);
        // the stage has landed for everyone, and everyone is done with the stage before
        if (!__syncthreads_and(ok)) {
            if (tid == 0)
                for (int q = st; q < issued; ++q) mbar_wait(bar0 + 8u * (q % STAGES), (q / STAGES) & 1, a.error, 34);
            return;
        }
        if (issued < stages) issue(issued++);
        const int ts = t0 + st * TOK;
        const float* stage = sd_sm + (size_t)(st % STAGES) * (TOK * ROW);
        const int n = min(TOK, t1 - ts);
        float o[NV];
#pragma unroll
        for (int tt = 0; tt < TOK; ++tt) {
            const float* row = stage + tt * ROW;
            F2 v[C], p[C][2], d[C];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                v[c].f.x = v[c].f.y = row[4 * DP + min(col + c, DP - 1)];
                p[c][0].f.x = p[c][0].f.y = p[c][1].f.x = p[c][1].f.y = d[c].f.x = d[c].f.y = 0.f;
            }
            // the sums over the old state
            union Four { float4 f; F2 p[2]; };
            Four u[RPT / 4];
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
                const int ch = i4 * SPLIT + part;
                Four rw;
                rw.f = reinterpret_cast<const float4*>(row)[ch];
                u[i4].f = reinterpret_cast<const float4*>(row + DP)[ch];
#pragma unroll
                for (int c = 0; c < C; ++c)
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        p[c][q] = fma2(s[c][i4 * 2 + q], u[i4].p[q], p[c][q]);
                        d[c] = fma2(s[c][i4 * 2 + q], rw.p[q], d[c]);
                    }
            }
            float ps[C];
#pragma unroll
            for (int c = 0; c < C; ++c) ps[c] = (p[c][0].f.x + p[c][1].f.x) + (p[c][0].f.y + p[c][1].f.y);
#pragma unroll
            for (int o2 = 1; o2 < SPLIT; o2 <<= 1)
#pragma unroll
                for (int c = 0; c < C; ++c) ps[c] += __shfl_xor_sync(0xffffffffu, ps[c], o2);
            const float rau = row[5 * DP], ru = row[5 * DP + 1];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                o[tt * C + c] = d[c].f.x + d[c].f.y;
                if (part == 0) o[tt * C + c] += rau * ps[c] + ru * v[c].f.x;
                p[c][0].f.x = p[c][0].f.y = ps[c];
            }
            // the new state
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
                const int ch = i4 * SPLIT + part;
                Four w, na;
                w.f = reinterpret_cast<const float4*>(row + 2 * DP)[ch];
                na.f = reinterpret_cast<const float4*>(row + 3 * DP)[ch];
#pragma unroll
                for (int c = 0; c < C; ++c)
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        F2& si = s[c][i4 * 2 + q];
                        si = fma2(na.p[q], p[c][0], fma2(si, w.p[q], mul2(u[i4].p[q], v[c])));
                    }
            }
        }
        // sum over the column's lanes: at every step a lane hands half of its values over and keeps the other half
#pragma unroll
        for (int step = SPLIT / 2, left = NV; step > 0; step >>= 1) {
            left >>= 1;
            const bool upper = (part & step) != 0;
#pragma unroll
            for (int j = 0; j < NV / 2; ++j) {
                if (j >= left) break;
                const float give = upper ? o[j] : o[j + left], keep = upper ? o[j + left] : o[j];
                o[j] = keep + __shfl_xor_sync(0xffffffffu, give, step);
            }
        }
#pragma unroll
        for (int j = 0; j < NV / SPLIT; ++j) {
            const int idx = part * (NV / SPLIT) + j, tt = idx / C, c = idx % C;
            if (tt < n && col + c < dim) a.out[((size_t)(ts + tt) * H + h) * dim + col + c] = o[j];
        }
    }
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
        for (int i = 0; i < RPT / 2; ++i) {
            const int r = ((i >> 1) * SPLIT + part) * 4 + (i & 1) * 2;
            if (col + c < dim) {
                if (r < dim) S[(size_t)r * dim + col + c] = s[c][i].f.x;
                if (r + 1 < dim) S[(size_t)(r + 1) * dim + col + c] = s[c][i].f.y;
            }
        }
}

template <int RPT, int SPLIT, int C, int THREADS, int TOK, int STAGES>
static int split_delta_scan_go(const SplitDeltaScanArgs& a, int B, bool early, cudaStream_t s) {
    constexpr int COLS = THREADS / SPLIT * C;
    constexpr size_t smem = (size_t)STAGES * TOK * (5 * RPT * SPLIT + 4) * sizeof(float);
    static_assert(smem <= 220 * 1024, "the stages fit an SM");
    static bool configured = false;
    if (smem > 48 * 1024 && !configured) {
        cudaError_t e = cudaFuncSetAttribute(split_delta_scan_kernel<RPT, SPLIT, C, THREADS, TOK, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    dim3 grid(B, a.H, (a.dim + COLS - 1) / COLS);
    if (early)
        TB_LAUNCH((split_delta_scan_kernel<RPT, SPLIT, C, THREADS, TOK, STAGES>), grid, THREADS, smem, s, a);
    else        // prompts: the blocks run for the whole sequence and want an SM each (see tb_launch_plain)
        tb_launch_plain(split_delta_scan_kernel<RPT, SPLIT, C, THREADS, TOK, STAGES>, grid, dim3(THREADS), smem, s, a);
    return tb_last_error();
}

static int split_delta_scan_launch(SplitDeltaScanArgs a, int B, cudaStream_t s) {
    if (B < 0 || a.H <= 0 || a.dim <= 0 || a.pitch < (long long)a.H * a.dim * a.dim) return TB_ERR_ARG;
    if (a.dim > 256) return TB_ERR_UNSUPPORTED;
    if (B == 0) return 0;
    a.error = tc_error_ptr();
    if (!a.error) return tb_last_error();
    const bool early = a.nt <= 2 * B;
    // Few columns of state in the batch: small pieces per thread, so that as many warps as there are keep the chain of a
    // token short (one prompt of 2,048 tokens: 16 heads of 128 387 us with 4 rows of 2 columns and 256 threads, 492 with 16
    // rows of 1 and 128; 8 heads of 128 324 us with 4 of 2 and 128 threads; 32 heads of 64 304 us with 4 of 1, 360 with 8 of
    // 1).  Enough of them to fill the GPU: larger pieces, which read a record's entry for more columns (eight prompts of 512
    // tokens: 16 heads of 128 371 us with 16 rows of 2, 707 with 4 of 2; 32 heads of 64 190 us with 8 of 4, 401 with 8 of 1).
    const long long columns = (long long)B * a.H * a.dim;
    const bool many = columns >= 128 * 32;
    switch (dm_rows(a.dim)) {
        case 16: return split_delta_scan_go<4, 4, 1, 128, 8, 4>(a, B, early, s);
        case 32: return split_delta_scan_go<4, 8, 1, 128, 8, 4>(a, B, early, s);
        case 64:
            return many ? split_delta_scan_go<8, 8, 4, 64, 8, 4>(a, B, early, s) : split_delta_scan_go<4, 16, 1, 128, 16, 3>(a, B, early, s);
        case 128:
            return many              ? split_delta_scan_go<16, 8, 2, 128, 8, 4>(a, B, early, s)
                   : columns > 1024 ? split_delta_scan_go<4, 32, 2, 256, 16, 3>(a, B, early, s)
                                    : split_delta_scan_go<4, 32, 2, 128, 16, 3>(a, B, early, s);
        default: return split_delta_scan_go<16, 16, 1, 128, 16, 2>(a, B, early, s);
    }
}

// ---- one token per sequence -------------------------------------------------------------------------------------
struct SplitDeltaStepArgs {
    const void* z;          // [nt, ldz]: r | k | v | gate
    const float* az;        // [nt, lda]: the removal rate's pre-activation, [H dim], then x1, [rank]
    const float* ba;
    const void* w2;         // [H dim, rank]
    const float* w0;
    const float* norm;      // [H dim]
    float* state;
    void* y;                // [nt, ldy]
    const int* seq_start;
    const int* slots;
    long long pitch;
    int nt, ldz, lda, ldy, H, dim, rank;
    float eps;
};

__host__ __device__ inline int sd_groups(int dim, int v) {      // groups of rows of a step block
    const int g = SD_STEP / (dim / v);
    return g < dim ? g : dim;
}

// V columns a thread and access; NR: rows a thread at most.
template <typename T, int V, int NR>
__global__ void __launch_bounds__(SD_STEP) split_delta_step_kernel(const SplitDeltaStepArgs p) {
    extern __shared__ __align__(16) float sd_sm[];
    const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int dim = p.dim, hd = p.H * dim, rank4 = (p.rank + 3) / 4 * 4, dim4 = (dim + 3) / 4 * 4;
    const int nc = dim / V, G = sd_groups(dim, V);
    float* ta = sd_sm;                      // [rank4]
    float* rw_s = ta + rank4;               // [dim4] each
    float* u_s = rw_s + dim4;
    float* w_s = u_s + dim4;
    float* na_s = w_s + dim4;
    float* v_s = na_s + dim4;
    float* p_s = v_s + dim4;
    float* part_p = p_s + dim4;             // [G][dim4] each
    float* part_q = part_p + G * dim4;
    __shared__ float red[33];
    const int hc = h * dim + tid;
    float nw = 0.f, ba = 0.f;
    if (tid < dim) {                        // weights: nothing of the step writes them
        nw = p.norm[hc];
        ba = p.ba[hc];
    }
    pdl_sync();
    const int t = p.seq_start[b];
    float* S = p.state + (size_t)p.slots[b] * p.pitch + (size_t)h * dim * dim;
    const T* z = static_cast<const T*>(p.z) + (size_t)t * p.ldz;
    // the state is on its way while everything else is made
    const int rg = tid / nc, c = (tid - rg * nc) * V;
    float s[NR][V];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int r = rg + i * G;
        if (rg < G && r < dim) dm_load<float, V>(S + (size_t)r * dim + c, s[i]);
    }
    for (int q = tid; q < p.rank; q += SD_STEP) ta[q] = tanhf(p.az[(size_t)t * p.lda + hd + q]);
    float r = 0.f, k = 0.f, v = 0.f, gate = 0.f, a = 0.f;
    if (tid < dim) {
        r = ldf(z + hc);
        k = ldf(z + hd + hc);
        v = ldf(z + 2 * hd + hc);
        gate = ldf(z + 3 * hd + hc);
        a = sd_sigmoid(p.az[(size_t)t * p.lda + hc] + ba);
    }
    const float len = sqrtf(block_sum(k * k, red) + SD_UNIT_EPS), u = k / len, vl = v * len;
    {
        // adjacent lanes share a channel's row of W2
        const int parts = SD_STEP / dm_rows(dim), ch = tid / parts, part = tid - ch * parts;
        float acc = 0.f;
        if (ch < dim)
            acc = decay_dot<T>(static_cast<const T*>(p.w2) + (size_t)(h * dim + ch) * p.rank, ta, p.rank, part, parts);
        for (int o = min(parts, 32) >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (ch < dim && part == 0) w_s[ch] = sd_decay(acc + p.w0[h * dim + ch]);
    }
    if (tid < dim) {
        u_s[tid] = u;
        na_s[tid] = -a * u;
        v_s[tid] = vl;
    }
    const float rau = block_sum(-r * a * u, red), ru = block_sum(r * u, red);       // (and everyone's part of w_s is there)
    if (tid < dim) rw_s[tid] = r * w_s[tid];
    __syncthreads();
    if (rg < G) {
        float ap[V], aq[V];
#pragma unroll
        for (int e = 0; e < V; ++e) ap[e] = aq[e] = 0.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int rr = rg + i * G;
            if (rr >= dim) break;
            const float ur = u_s[rr], wr = rw_s[rr];
#pragma unroll
            for (int e = 0; e < V; ++e) {
                ap[e] += s[i][e] * ur;
                aq[e] += s[i][e] * wr;
            }
        }
        dm_store<V>(part_p + rg * dim4 + c, ap);
        dm_store<V>(part_q + rg * dim4 + c, aq);
    }
    __syncthreads();
    float o = 0.f;
    if (tid < dim) {
        float pj = 0.f;
        for (int g = 0; g < G; ++g) {
            pj += part_p[g * dim4 + tid];
            o += part_q[g * dim4 + tid];
        }
        o += rau * pj + ru * vl;
        p_s[tid] = pj;
    }
    __syncthreads();
    if (rg < G) {
        float pc[V], vc[V];
        dm_load<float, V>(p_s + c, pc);
        dm_load<float, V>(v_s + c, vc);
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int rr = rg + i * G;
            if (rr >= dim) break;
            const float ur = u_s[rr], wr = w_s[rr], nr = na_s[rr];
#pragma unroll
            for (int e = 0; e < V; ++e) s[i][e] = s[i][e] * wr + nr * pc[e] + ur * vc[e];
            dm_store<V>(S + (size_t)rr * dim + c, s[i]);
        }
    }
    const float rs = 1.0f / sqrtf(block_sum(o * o, red) / (float)dim + p.eps);
    if (tid < dim) stf(static_cast<T*>(p.y) + (size_t)t * p.ldy + hc, o * rs * nw * sd_sigmoid(gate));
}

template <typename T>
static int split_delta_step_launch(const SplitDeltaStepArgs& p, int B, cudaStream_t s) {
    if (B < 0 || p.nt < B || p.H <= 0 || p.dim <= 0 || p.rank <= 0 || p.lda < p.H * p.dim + p.rank || p.ldz < 4 * p.H * p.dim ||
        p.ldy < p.H * p.dim || p.pitch < (long long)p.H * p.dim * p.dim)
        return TB_ERR_ARG;
    if (p.dim > 128 || p.rank > 4096 || (p.rank % 8 == 0 && ((uintptr_t)p.w2 & 15))) return TB_ERR_UNSUPPORTED;
    if (B == 0) return 0;
    const bool vec = p.dim % 4 == 0 && p.pitch % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
    const int dim4 = (p.dim + 3) / 4 * 4, G = sd_groups(p.dim, vec ? 4 : 1);
    const size_t smem = ((size_t)(p.rank + 3) / 4 * 4 + (size_t)(6 + 2 * G) * dim4) * sizeof(float);
    if (smem > 48 * 1024) return TB_ERR_UNSUPPORTED;
    if (vec) TB_LAUNCH((split_delta_step_kernel<T, 4, 8>), dim3(B, p.H), SD_STEP, smem, s, p);
    else TB_LAUNCH((split_delta_step_kernel<T, 1, 32>), dim3(B, p.H), SD_STEP, smem, s, p);
    return tb_last_error();
}

extern "C" {
int tb_split_delta_record_size(int dim) { return sd_record(dim); }
#define TB_SPLIT_DELTA(SFX, T)                                                                                        \
    int tb_split_delta_prep_##SFX(const void* z, int ldz, const float* az, int lda, const float* ba,                  \
                                  const float* pre, const float* w0, float* rec, int nt, int H, int dim,              \
                                  cudaStream_t s) {                                                                   \
        if ((uintptr_t)rec & 15) return TB_ERR_ARG;                                                                   \
        return split_delta_prep_launch<T>(SplitDeltaArgs{z, az, ba, pre, w0, rec, nt, ldz, lda, H, dim}, s);          \
    }                                                                                                                 \
    int tb_split_delta_step_##SFX(const void* z, int ldz, const float* az, int lda, const float* ba, const void* w2,  \
                                  const float* w0, const float* norm, float eps, float* state, long long pitch,       \
                                  void* y, int ldy, const int* seq_start, const int* slots, int nt, int B, int H,     \
                                  int dim, int rank, cudaStream_t s) {                                                \
        return split_delta_step_launch<T>(SplitDeltaStepArgs{z, az, ba, w2, w0, norm, state, y, seq_start, slots,     \
                                                             pitch, nt, ldz, lda, ldy, H, dim, rank, eps}, B, s);     \
    }
TB_SPLIT_DELTA(f32, float)
TB_SPLIT_DELTA(bf16, __nv_bfloat16)

int tb_split_delta_scan(const float* rec, float* state, long long pitch, float* out, const int* seq_start,
                        const int* slots, int nt, int B, int H, int dim, cudaStream_t s) {
    if ((uintptr_t)rec & 15) return TB_ERR_ARG;
    return split_delta_scan_launch(SplitDeltaScanArgs{rec, state, nullptr, out, seq_start, slots, pitch, nt, H, dim}, B, s);
}
}

#include "tape.h"
TB_TAPE_REGISTER(tb_split_delta_prep_f32)
TB_TAPE_REGISTER(tb_split_delta_prep_bf16)
TB_TAPE_REGISTER(tb_split_delta_step_f32)
TB_TAPE_REGISTER(tb_split_delta_step_bf16)
TB_TAPE_REGISTER(tb_split_delta_scan)
