// A linear memory with a decay per key channel made from the input, a bonus for the current token and a shift of the
// input by one token (the time mixing of the RWKV family), state in float.
//
// Per head, with a state S [dim, dim] that is zero when a sequence starts (rows: key channels, columns: values):
//
//   o_t = S^T r_t + (r_t . (u k_t)) v_t;        S <- diag(w_t) S + k_t v_t^T;        w = exp(-exp(w0 + W2 tanh(a)))
//
// r, k, v, a and the output gate are projections of mixes of the token's input and the input of the token before:
//   mix_m[t] = x[t] + (x[t - 1] - x[t]) mu_m        x[-1]: the sequence's last input of the step before (zeros at its start)
//
// State of one slot (floats): S [H][dim][dim], then the last input [width]; the pitch is a multiple of four.
//
//   shift_mix_kernel    all mixes of a token at once, and the group lists of the product that follows (a matrix per mix)
//   decay_tanh_kernel   prompts: tanh(a) for the product with W2
//   decay_prep_kernel   prompts: decays and bonuses; one float record per (token, head) for the scan, r | k | w | v | bonus,
//                       those of a head one behind the other
//   decay_scan_kernel   prompts: the recurrence token by token, a block = a sequence x a head x some columns of S, whose
//                       rows are split over adjacent lanes, in registers; the lanes' sums meet only in the output, so
//                       no token waits for another's reduction
//                       (also the scan of a memory [dim, vdim] that is read after it is written to: csrc/gated_linear.cu)
//   decay_step_kernel   one token per sequence: a block = a sequence x a head; decays, bonus, the state's way through the
//                       registers, the head's norm and the gate in one kernel
// Everything that enters the recurrence is float on both paths; x, r, k, v and the gate have the activations' type.
#include "memory_common.cuh"
#include "tc_common.cuh"                // bulk copies, barriers with bounded waits

constexpr int DM_MIXES = 5;             // r, k, v, gate, decay
constexpr int DM_SCAN = 128;            // threads of a scan block

// floats of a record's values (16-byte pieces), and of a record, r | k | w | v | bonus, 0, 0, 0
__host__ __device__ inline int dm_values(int dim, int vdim) { return vdim == dim ? dm_rows(dim) : (vdim + 3) / 4 * 4; }
__host__ __device__ inline int dm_record(int dim, int vdim) { return 3 * dm_rows(dim) + dm_values(dim, vdim) + 4; }
__host__ __device__ inline long long dm_state(int H, int dim, int width) { return ((long long)H * dim * dim + width + 3) / 4 * 4; }

// ---- the mixes ---------------------------------------------------------------------------------------------
template <typename T, bool VEC, int TILE>
__global__ void __launch_bounds__(128)
shift_mix_kernel(const T* __restrict__ x, const float* __restrict__ mu, const float* __restrict__ state,
                 long long pitch, long long at, T* __restrict__ out, int* __restrict__ offsets,
                 int* __restrict__ row_group, int groups, const int* __restrict__ tok_seq,
                 const int* __restrict__ seq_start, const int* __restrict__ slots, int nt, int d) {
    constexpr int V = VEC ? 8 : 1;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    float m[DM_MIXES][V];
#pragma unroll
    for (int j = 0; j < DM_MIXES; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) m[j][e] = 0.f;
    if (c < d) {        // weights: nothing of the step writes them
#pragma unroll
        for (int j = 0; j < DM_MIXES; ++j) {
            if constexpr (VEC) load8(mu + (size_t)j * d + c, m[j]);
            else m[j][0] = mu[(size_t)j * d + c];
        }
    }
    pdl_sync();
    if (blockIdx.x == 0 && blockIdx.y == 0) {
        for (int j = threadIdx.x; j <= groups; j += blockDim.x) offsets[j] = j * nt;
        if (row_group)
            for (int j = threadIdx.x; j < groups * nt; j += blockDim.x) row_group[j] = j / nt;
    }
    if (c >= d) return;
    const int t0 = blockIdx.x * TILE;
    float before[V], now[V];
#pragma unroll
    for (int tt = 0; tt < TILE; ++tt) {
        const int t = t0 + tt;
        if (t >= nt) break;
        const int b = tok_seq[t];
        if constexpr (VEC) load8(x + (size_t)t * d + c, now);
        else now[0] = ldf(x + (size_t)t * d + c);
        if (t == seq_start[b]) {
            const float* last = state + (size_t)slots[b] * pitch + at + c;
#pragma unroll
            for (int e = 0; e < V; ++e) before[e] = last[e];
        } else if (tt == 0) {
            if constexpr (VEC) load8(x + (size_t)(t - 1) * d + c, before);
            else before[0] = ldf(x + (size_t)(t - 1) * d + c);
        }
#pragma unroll
        for (int j = 0; j < DM_MIXES; ++j) {
            float y[V];
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = now[e] + (before[e] - now[e]) * m[j][e];
            T* dst = out + ((size_t)j * nt + t) * d + c;
            if constexpr (VEC) store8(dst, y);
            else stf(dst, y[0]);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) before[e] = now[e];
    }
}

template <typename T>
static int shift_mix_launch(const void* x, const float* mu, const float* state, long long pitch, long long at, void* out,
                            int* offsets, int* row_group, int groups, const int* tok_seq, const int* seq_start,
                            const int* slots, int nt, int d, cudaStream_t s) {
    if (nt < 0 || d <= 0 || groups < 1 || !offsets) return TB_ERR_ARG;
    if (nt == 0) return 0;
    const bool vec = d % 8 == 0 && (((uintptr_t)x | (uintptr_t)mu | (uintptr_t)out) & 15) == 0;
    const int per = 128 * (vec ? 8 : 1), cols = (d + per - 1) / per;
    const bool tiled = nt >= 256;
    const dim3 grid(tiled ? (nt + 3) / 4 : nt, cols);
#define SHIFT_GO(VEC, TILE)                                                                                           \
    TB_LAUNCH((shift_mix_kernel<T, VEC, TILE>), grid, 128, 0, s, (const T*)x, mu, state, pitch, at, (T*)out, offsets, \
              row_group, groups, tok_seq, seq_start, slots, nt, d)
    if (vec && tiled) SHIFT_GO(true, 4);
    else if (vec) SHIFT_GO(true, 1);
    else if (tiled) SHIFT_GO(false, 4);
    else SHIFT_GO(false, 1);
#undef SHIFT_GO
    return tb_last_error();
}

// ---- decays ------------------------------------------------------------------------------------------------
// tanh of the decay's first projection, ready for the product with W2: in the activations' type a value is stored as the
// sum of two (what its rounding leaves goes into the second half of the row, and the product's weight holds W2 twice), so
// the product loses nothing that matters; in float it is stored as it is.  plain: the projection itself, without tanh.
template <typename T>
__global__ void __launch_bounds__(256) decay_tanh_kernel(const float* __restrict__ a, int lda, T* __restrict__ out, int nt,
                                                         int rank, int ldo, int plain) {
    pdl_sync();
    const int n = nt * ldo;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
        const int t = i / ldo, q = i - t * ldo;
        const int half = sizeof(T) == 2 ? ldo / 2 : ldo;        // entries of a half, beyond rank zero
        const int e = q < half ? q : q - half;
        float v = 0.f;
        if (e < rank) {
            v = a[(size_t)t * lda + e];
            if (!plain) v = tanhf(v);
            if (q >= half) {
                T hi;
                stf(&hi, v);
                v -= ldf(&hi);
            }
        }
        stf(out + i, v);
    }
}

struct DecayArgs {
    const void* z;          // [4 nt, H dim]: r, k, v, gate, nt rows each
    const float* pre;       // [nt, H dim]  W2 tanh(.)
    const float* w0;        // [H dim]
    const float* u;         // [H dim]
    float* rec;             // [H, nt, dm_record]
    int nt, H, dim;
};

// A warp per (token, head): the record and the values; four neighbouring entries a lane and access where the layout
// allows it (VEC).
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) decay_prep_kernel(const DecayArgs p) {
    pdl_sync();
    constexpr int V = VEC ? 4 : 1;
    const int lane = threadIdx.x & 31;
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (row >= p.nt * p.H) return;
    const int t = row / p.H, h = row - t * p.H, dim = p.dim, hd = p.H * dim;
    const int DP = dm_rows(dim);
    float* rec = p.rec + ((size_t)h * p.nt + t) * dm_record(dim, dim);
    const T* z = static_cast<const T*>(p.z) + (size_t)t * hd + h * dim;
    const size_t part = (size_t)p.nt * hd;
    float bonus = 0.f;
    for (int c = lane * V; c < DP; c += 32 * V) {
        float r[V], k[V], v[V], w[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            r[e] = k[e] = v[e] = 0.f;
            w[e] = 1.f;
        }
        if (c < dim) {
            float pre[V], w0[V], u[V];
            dm_load<T, V>(z + c, r);
            dm_load<T, V>(z + part + c, k);
            dm_load<T, V>(z + 2 * part + c, v);
            dm_load<float, V>(p.pre + (size_t)t * hd + h * dim + c, pre);
            dm_load<float, V>(p.w0 + h * dim + c, w0);
            dm_load<float, V>(p.u + h * dim + c, u);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                w[e] = expf(-expf(pre[e] + w0[e]));
                bonus += r[e] * u[e] * k[e];
            }
        }
        dm_store<V>(rec + c, r);
        dm_store<V>(rec + DP + c, k);
        dm_store<V>(rec + 2 * DP + c, w);
        dm_store<V>(rec + 3 * DP + c, v);
    }
    bonus = warp_sum(bonus);
    if (lane < 4) rec[4 * DP + lane] = lane == 0 ? bonus : 0.f;
}

// ---- the scan ------------------------------------------------------------------------------------------------
struct DecayScanArgs {
    const float* rec;
    float* state;           // [slots, pitch]
    int* error;             // set by a wait that runs out
    float* out;             // [nt, H dim]
    const void* x;          // [nt, width]: a sequence's last row becomes its state's last input (null: there is none)
    const int* seq_start;
    const int* slots;
    long long pitch;
    int nt, H, dim, width, vdim;
};

// RPT rows of C columns per thread, SPLIT lanes per column (SPLIT * RPT = dm_rows(dim)): DM_SCAN / SPLIT * C columns a
// block.  The records of TOK tokens at a time are one bulk copy to shared memory, STAGES - 1
// stages ahead.  A
// token needs no reduction: every lane keeps its rows' share of the outputs of a whole stage, and the TOK * C shares
// are then summed over the column's lanes so that each lane ends with some of the sums (fewer shuffles than sums).
// SQUARE: vdim equals dim (a record's length is then known when this is compiled).
template <typename T, int RPT, int SPLIT, int C, int TOK, int STAGES, bool SQUARE>
__global__ void __launch_bounds__(DM_SCAN) decay_scan_kernel(const DecayScanArgs a) {
    pdl_sync();
    constexpr int DP = RPT * SPLIT;
    constexpr int COLS = DM_SCAN / SPLIT * C;
    const int VP = SQUARE ? DP : dm_values(a.dim, a.vdim);
    const int ROW = 3 * DP + VP + 4;                    // a record
    constexpr int NV = TOK * C;
    static_assert(NV % SPLIT == 0, "every lane ends with as many sums");
    extern __shared__ __align__(16) float dm_sm[];      // [STAGES][TOK][ROW]
    __shared__ __align__(8) unsigned long long bars[STAGES];
    const int b = blockIdx.x, h = blockIdx.y;
    const int tid = threadIdx.x, part = tid & (SPLIT - 1), cl = tid / SPLIT * C;
    const int col0 = blockIdx.z * COLS, col = col0 + cl;
    const int dim = a.dim, vdim = SQUARE ? dim : a.vdim, H = a.H;
    const int t0 = a.seq_start[b], t1 = a.seq_start[b + 1];
    if (t0 >= t1) return;
    float* slot = a.state + (size_t)a.slots[b] * a.pitch;
    float* S = slot + (size_t)h * dim * vdim;
    F2 s[C][RPT / 2];                                   // rows 2i, 2i + 1 of this lane's
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
        for (int i = 0; i < RPT / 2; ++i) {
            const int r = ((i >> 1) * SPLIT + part) * 4 + (i & 1) * 2;
            s[c][i].f.x = (r < dim && col + c < vdim) ? S[(size_t)r * vdim + col + c] : 0.f;
            s[c][i].f.y = (r + 1 < dim && col + c < vdim) ? S[(size_t)(r + 1) * vdim + col + c] : 0.f;
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
        float* to = dm_sm + (size_t)(q % STAGES) * (TOK * ROW);
        if (tid == 0) {
            const uint32_t bytes = (uint32_t)(n * ROW) * sizeof(float);
            mbar_expect_tx(bar0 + 8u * (q % STAGES), bytes);
            bulk_load(smem_u32(to), rec + (size_t)ts * ROW, bytes, bar0 + 8u * (q % STAGES));
        }
        // tokens behind the last: nothing is written, nothing fades, nothing is read (so that a stage has no branches)
        for (int idx = n * ROW + tid; idx < TOK * ROW; idx += DM_SCAN) {
            const int e = idx % ROW;
            to[idx] = e >= 2 * DP && e < 3 * DP ? 1.f : 0.f;
        }
    };
    int issued = 0;
    for (; issued < STAGES - 1 && issued < stages; ++issued) issue(issued);
    for (int st = 0; st < stages; ++st) {
        const bool ok = mbar_wait(bar0 + 8u * (st % STAGES), (st / STAGES) & 1, a.error, 31);
        // the stage has landed for everyone, and everyone is done with the stage before
        if (!__syncthreads_and(ok)) {
            if (tid == 0)
                for (int q = st; q < issued; ++q) mbar_wait(bar0 + 8u * (q % STAGES), (q / STAGES) & 1, a.error, 32);
            return;
        }
        if (issued < stages) issue(issued++);
        const int ts = t0 + st * TOK;
        const float* stage = dm_sm + (size_t)(st % STAGES) * (TOK * ROW);
        const int n = min(TOK, t1 - ts);
        float o[NV];
#pragma unroll
        for (int tt = 0; tt < TOK; ++tt) {
            const float* row = stage + tt * ROW;
            F2 v[C], d[C];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                v[c].f.x = v[c].f.y = row[3 * DP + min(col + c, VP - 1)];
                d[c].f.x = d[c].f.y = 0.f;
            }
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
                const int ch = i4 * SPLIT + part;
                union { float4 f; F2 p[2]; } r, k, w;
                r.f = reinterpret_cast<const float4*>(row)[ch];
                k.f = reinterpret_cast<const float4*>(row + DP)[ch];
                w.f = reinterpret_cast<const float4*>(row + 2 * DP)[ch];
#pragma unroll
                for (int c = 0; c < C; ++c)
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        F2& si = s[c][i4 * 2 + q];
                        d[c] = fma2(si, r.p[q], d[c]);
                        si = fma2(si, w.p[q], mul2(k.p[q], v[c]));
                    }
            }
#pragma unroll
            for (int c = 0; c < C; ++c) o[tt * C + c] = d[c].f.x + d[c].f.y;
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
            if (tt < n && col + c < vdim) {
                const float* row = stage + tt * ROW;
                a.out[((size_t)(ts + tt) * H + h) * vdim + col + c] = o[j] + row[3 * DP + VP] * row[3 * DP + col + c];
            }
        }
    }
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
        for (int i = 0; i < RPT / 2; ++i) {
            const int r = ((i >> 1) * SPLIT + part) * 4 + (i & 1) * 2;
            if (col + c < vdim) {
                if (r < dim) S[(size_t)r * vdim + col + c] = s[c][i].f.x;
                if (r + 1 < dim) S[(size_t)(r + 1) * vdim + col + c] = s[c][i].f.y;
            }
        }
    if (h == 0 && blockIdx.z == 0 && a.x) {        // the mixes have read the old one
        const T* last = static_cast<const T*>(a.x) + (size_t)(t1 - 1) * a.width;
        float* to = slot + (size_t)H * dim * dim;
        for (int c = tid; c < a.width; c += DM_SCAN) to[c] = ldf(last + c);
    }
}

template <typename T, bool SQUARE, int RPT, int SPLIT, int C, int TOK, int STAGES>
static int decay_scan_go(const DecayScanArgs& a, int B, bool early, cudaStream_t s) {
    constexpr int COLS = DM_SCAN / SPLIT * C;
    const size_t smem = (size_t)STAGES * TOK * dm_record(a.dim, a.vdim) * sizeof(float);
    if (smem > 220 * 1024) return TB_ERR_UNSUPPORTED;
    static size_t configured = 48 * 1024;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(decay_scan_kernel<T, RPT, SPLIT, C, TOK, STAGES, SQUARE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = smem;
    }
    dim3 grid(B, a.H, (a.vdim + COLS - 1) / COLS);
    if (early)
        TB_LAUNCH((decay_scan_kernel<T, RPT, SPLIT, C, TOK, STAGES, SQUARE>), grid, DM_SCAN, smem, s, a);
    else        // prompts: the blocks run for the whole sequence and want an SM each (see tb_launch_plain)
        tb_launch_plain(decay_scan_kernel<T, RPT, SPLIT, C, TOK, STAGES, SQUARE>, grid, dim3(DM_SCAN), smem, s, a);
    return tb_last_error();
}

template <typename T, bool SQUARE>
static int decay_scan_launch(DecayScanArgs a, int B, cudaStream_t s) {
    if (B < 0 || a.H <= 0 || a.dim <= 0 || a.vdim <= 0 || a.pitch < (long long)a.H * a.dim * a.vdim) return TB_ERR_ARG;
    if (a.x && (a.width <= 0 || a.vdim != a.dim || a.pitch < dm_state(a.H, a.dim, a.width))) return TB_ERR_ARG;
    if (a.dim > 256) return TB_ERR_UNSUPPORTED;
    if (B == 0) return 0;
    a.error = tc_error_ptr();
    if (!a.error) return tb_last_error();
    const bool early = a.nt <= 2 * B;
    // Few sequences: small pieces of the state per thread, so that as many warps as there are keep the chain of a token
    // short (16 heads of 128, one prompt of 2,048 tokens: 197 us with 4 rows of 2 columns, 245 with 8 of 2, 320 with 8
    // of 4).  Enough of them to fill the GPU: larger pieces, which read a record's entry for more columns (eight
    // prompts of 1,024 tokens: 444 us with 8 rows of 4 columns, 665 with 4 of 2).
    const bool many = (long long)B * a.H * a.vdim >= 128 * 32;
    switch (dm_rows(a.dim)) {
        case 16: return decay_scan_go<T, SQUARE, 4, 4, 1, 8, 4>(a, B, early, s);
        case 32: return decay_scan_go<T, SQUARE, 4, 8, 1, 8, 4>(a, B, early, s);
        case 64:
            return many ? decay_scan_go<T, SQUARE, 8, 8, 4, 8, 4>(a, B, early, s) : decay_scan_go<T, SQUARE, 4, 16, 2, 16, 3>(a, B, early, s);
        case 128:
            return many ? decay_scan_go<T, SQUARE, 8, 16, 4, 8, 4>(a, B, early, s) : decay_scan_go<T, SQUARE, 4, 32, 2, 16, 3>(a, B, early, s);
        default: return decay_scan_go<T, SQUARE, 8, 32, 4, 8, 3>(a, B, early, s);
    }
}

template <typename T>
static int decay_prep_launch(const DecayArgs& p, cudaStream_t s) {
    if (p.nt < 0 || p.H <= 0 || p.dim <= 0) return TB_ERR_ARG;
    if (p.dim > 256) return TB_ERR_UNSUPPORTED;
    if (p.nt == 0) return 0;
    const bool vec = p.dim % 4 == 0 &&
                     (((uintptr_t)p.z | (uintptr_t)p.pre | (uintptr_t)p.w0 | (uintptr_t)p.u) & 15) == 0;
    const int grid = (int)(((long long)p.nt * p.H + 7) / 8);
    if (vec) TB_LAUNCH((decay_prep_kernel<T, true>), grid, 256, 0, s, p);
    else TB_LAUNCH((decay_prep_kernel<T, false>), grid, 256, 0, s, p);
    return tb_last_error();
}
template <typename T>
static int decay_tanh_launch(const float* a, int lda, void* out, int nt, int rank, int ldo, int plain, cudaStream_t s) {
    if (nt < 0 || rank <= 0 || lda < rank || ldo < rank * (sizeof(T) == 2 ? 2 : 1) || (sizeof(T) == 2 && ldo % 2)) return TB_ERR_ARG;
    if (nt == 0) return 0;
    const long long n = (long long)nt * ldo;
    if (n > (1ll << 30)) return TB_ERR_UNSUPPORTED;
    TB_LAUNCH((decay_tanh_kernel<T>), (int)((n + 255) / 256 > 1184 ? 1184 : (n + 255) / 256), 256, 0, s, a, lda, (T*)out, nt, rank, ldo, plain);
    return tb_last_error();
}

// ---- one token per sequence -------------------------------------------------------------------------------------
struct DecayStepArgs {
    const void* z;          // [4 nt, H dim]: r, k, v, gate, nt rows each
    const void* x;          // [nt, width]
    const float* a;         // [nt, lda]
    const void* w2;
    const float* w0;
    const float* u;
    const float* norm;      // [H dim]
    float* state;
    void* y;                // [nt, ldy]
    const int* seq_start;
    const int* slots;
    long long pitch;
    int nt, width, lda, ldy, H, dim, rank;
    float eps;
};

// VEC: four columns a thread and access (dim a multiple of four), else one.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) decay_step_kernel(const DecayStepArgs p) {
    constexpr int V = VEC ? 4 : 1;
    constexpr int U = 8;                    // rows asked for together
    extern __shared__ __align__(16) float dm_sm[];
    const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int dim = p.dim, hd = p.H * dim, rank4 = (p.rank + 3) / 4 * 4, dim4 = (dim + 3) / 4 * 4;
    const int nc = dim / V, G = 256 / nc;   // columns' threads, groups of rows
    float* ta = dm_sm;                      // [rank4]
    float* r_s = ta + rank4;                // [dim4] each
    float* k_s = r_s + dim4;
    float* w_s = k_s + dim4;
    float* v_s = w_s + dim4;
    float* o_s = v_s + dim4;                // [G][dim4]
    __shared__ float red[33];
    const int hc = h * dim + tid;
    float u = 0.f, nw = 0.f;
    if (tid < dim) {                        // weights: nothing of the step writes them
        u = p.u[hc];
        nw = p.norm[hc];
    }
    pdl_sync();
    const int t = p.seq_start[b];
    float* slot = p.state + (size_t)p.slots[b] * p.pitch;
    float* S = slot + (size_t)h * dim * dim;
    const T* z = static_cast<const T*>(p.z);
    // the state's first rows are on their way while the decays are made
    const int rg = tid / nc, c = (tid - rg * nc) * V;
    float s[U][V];
    auto fetch = [&](int r0) {
#pragma unroll
        for (int q = 0; q < U; ++q) {
            const int r = r0 + q * G;
            if (r >= dim) continue;
            if constexpr (VEC) {
                const float4 f = *reinterpret_cast<const float4*>(S + (size_t)r * dim + c);
                s[q][0] = f.x; s[q][1] = f.y; s[q][2] = f.z; s[q][3] = f.w;
            } else {
                s[q][0] = S[(size_t)r * dim + c];
            }
        }
    };
    if (rg < G) fetch(rg);
    for (int q = tid; q < p.rank; q += 256) ta[q] = tanhf(p.a[(size_t)t * p.lda + q]);
    float bonus = 0.f, gate = 0.f;
    if (tid < dim) {
        const float r = ldf(z + (size_t)t * hd + hc), k = ldf(z + ((size_t)p.nt + t) * hd + hc);
        r_s[tid] = r;
        k_s[tid] = k;
        v_s[tid] = ldf(z + ((size_t)2 * p.nt + t) * hd + hc);
        gate = ldf(z + ((size_t)3 * p.nt + t) * hd + hc);
        bonus = r * u * k;
    }
    __syncthreads();
    {
        // adjacent lanes share a channel's row of W2
        const int parts = 256 / dm_rows(dim), ch = tid / parts, part = tid - ch * parts;
        float acc = 0.f;
        if (ch < dim)
            acc = decay_dot<T>(static_cast<const T*>(p.w2) + (size_t)(h * dim + ch) * p.rank, ta, p.rank, part, parts);
        for (int o = parts >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (ch < dim && part == 0) w_s[ch] = expf(-expf(acc + p.w0[h * dim + ch]));
    }
    bonus = block_sum(bonus, red);          // (and everyone's part of w_s is there)
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
                const float rr = r_s[r], kk = k_s[r], ww = w_s[r];
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    acc[e] += s[q][e] * rr;
                    s[q][e] = s[q][e] * ww + kk * v[e];
                }
                if constexpr (VEC)
                    *reinterpret_cast<float4*>(S + (size_t)r * dim + c) = make_float4(s[q][0], s[q][1], s[q][2], s[q][3]);
                else
                    S[(size_t)r * dim + c] = s[q][0];
            }
        }
#pragma unroll
        for (int e = 0; e < V; ++e) o_s[rg * dim4 + c + e] = acc[e];
    }
    __syncthreads();
    float o = 0.f;
    if (tid < dim) {
        for (int g = 0; g < G; ++g) o += o_s[g * dim4 + tid];
        o += bonus * v_s[tid];
    }
    const float rs = 1.0f / sqrtf(block_sum(o * o, red) / (float)dim + p.eps);
    if (tid < dim) stf(static_cast<T*>(p.y) + (size_t)t * p.ldy + hc, o * rs * nw * (gate / (1.0f + expf(-gate))));
    if (h == 0) {                           // the mixes have read the old one
        const T* row = static_cast<const T*>(p.x) + (size_t)t * p.width;
        float* to = slot + (size_t)p.H * dim * dim;
        for (int q = tid; q < p.width; q += 256) to[q] = ldf(row + q);
    }
}

template <typename T>
static int decay_step_launch(const DecayStepArgs& p, int B, cudaStream_t s) {
    if (B < 0 || p.nt < B || p.H <= 0 || p.dim <= 0 || p.rank <= 0 || p.lda < p.rank || p.ldy < p.H * p.dim ||
        p.pitch < dm_state(p.H, p.dim, p.width))
        return TB_ERR_ARG;
    if (p.dim > 256 || p.rank > 4096 || (p.rank % 8 == 0 && ((uintptr_t)p.w2 & 15))) return TB_ERR_UNSUPPORTED;
    if (B == 0) return 0;
    const bool vec = p.dim % 4 == 0 && p.pitch % 4 == 0 && ((uintptr_t)p.state & 15) == 0;
    const int dim4 = (p.dim + 3) / 4 * 4, G = 256 / (p.dim / (vec ? 4 : 1));
    const size_t smem = ((size_t)(p.rank + 3) / 4 * 4 + (size_t)(4 + G) * dim4) * sizeof(float);
    if (smem > 48 * 1024) return TB_ERR_UNSUPPORTED;
    if (vec) TB_LAUNCH((decay_step_kernel<T, true>), dim3(B, p.H), 256, smem, s, p);
    else TB_LAUNCH((decay_step_kernel<T, false>), dim3(B, p.H), 256, smem, s, p);
    return tb_last_error();
}

extern "C" {
// Floats of state per slot.
int tb_decay_state_size(int H, int dim, int width) { return (int)dm_state(H, dim, width); }
int tb_decay_record_size(int dim) { return dm_record(dim, dim); }
// The scan alone, of a memory [dim, vdim] per head that lies at the start of a slot's state; rec [H, nt, record size].
int tb_decay_scan_rect_record_size(int dim, int vdim) { return dm_record(dim, vdim); }
int tb_decay_scan_rect(const float* rec, float* state, long long pitch, float* out, const int* seq_start, const int* slots,
                       int nt, int B, int H, int dim, int vdim, cudaStream_t s) {
    if ((uintptr_t)rec & 15) return TB_ERR_ARG;
    const DecayScanArgs a{rec, state, nullptr, out, nullptr, seq_start, slots, pitch, nt, H, dim, 0, vdim};
    return vdim == dim ? decay_scan_launch<float, true>(a, B, s) : decay_scan_launch<float, false>(a, B, s);
}
// out [5, nt, d]: the mixes of every token; offsets [groups + 1] and row_group [groups nt] (may be null): the lists by
// which one grouped product multiplies the first `groups` of them with a matrix each.  `at`: where in a slot's state the
// last input lies.
#define TB_DECAY(SFX, T)                                                                                              \
    int tb_shift_mix_##SFX(const void* x, const float* mu, const float* state, long long pitch, long long at,         \
                           void* out, int* offsets, int* row_group, int groups, const int* tok_seq,                   \
                           const int* seq_start, const int* slots, int nt, int d, cudaStream_t s) {                   \
        return shift_mix_launch<T>(x, mu, state, pitch, at, out, offsets, row_group, groups, tok_seq, seq_start,      \
                                   slots, nt, d, s);                                                                  \
    }                                                                                                                 \
    int tb_decay_tanh_##SFX(const float* a, int lda, void* out, int nt, int rank, int ldo, cudaStream_t s) {          \
        return decay_tanh_launch<T>(a, lda, out, nt, rank, ldo, 0, s);                                                \
    }                                                                                                                 \
    int tb_split_rows_##SFX(const float* a, int lda, void* out, int nt, int rank, int ldo, cudaStream_t s) {          \
        return decay_tanh_launch<T>(a, lda, out, nt, rank, ldo, 1, s);                                                \
    }                                                                                                                 \
    int tb_decay_prep_##SFX(const void* z, const float* pre, const float* w0, const float* u, float* rec,             \
                            int nt, int H, int dim, cudaStream_t s) {                                                 \
        if ((uintptr_t)rec & 15) return TB_ERR_ARG;                                                                   \
        return decay_prep_launch<T>(DecayArgs{z, pre, w0, u, rec, nt, H, dim}, s);                              \
    }                                                                                                                 \
    int tb_decay_scan_##SFX(const float* rec, float* state, long long pitch, float* out, const void* x, int width,    \
                            const int* seq_start, const int* slots, int nt, int B, int H, int dim, cudaStream_t s) {  \
        if ((uintptr_t)rec & 15) return TB_ERR_ARG;                                                                   \
        if (!x) return TB_ERR_ARG;                                                                                    \
        return decay_scan_launch<T, true>(DecayScanArgs{rec, state, nullptr, out, x, seq_start, slots, pitch, nt, H,  \
                                                        dim, width, dim}, B, s);                                      \
    }                                                                                                                 \
    int tb_decay_step_##SFX(const void* z, const void* x, int width, const float* a, int lda, const void* w2,         \
                            const float* w0, const float* u, const float* norm, float eps, float* state,              \
                            long long pitch, void* y, int ldy, const int* seq_start, const int* slots, int nt, int B, \
                            int H, int dim, int rank, cudaStream_t s) {                                               \
        return decay_step_launch<T>(DecayStepArgs{z, x, a, w2, w0, u, norm, state, y, seq_start, slots, pitch, nt,    \
                                                  width, lda, ldy, H, dim, rank, eps}, B, s);                         \
    }
TB_DECAY(f32, float)
TB_DECAY(bf16, __nv_bfloat16)
}

#include "tape.h"
TB_TAPE_REGISTER(tb_shift_mix_f32)
TB_TAPE_REGISTER(tb_shift_mix_bf16)
TB_TAPE_REGISTER(tb_split_rows_f32)
TB_TAPE_REGISTER(tb_split_rows_bf16)
TB_TAPE_REGISTER(tb_decay_tanh_f32)
TB_TAPE_REGISTER(tb_decay_tanh_bf16)
TB_TAPE_REGISTER(tb_decay_prep_f32)
TB_TAPE_REGISTER(tb_decay_prep_bf16)
TB_TAPE_REGISTER(tb_decay_scan_f32)
TB_TAPE_REGISTER(tb_decay_scan_bf16)
TB_TAPE_REGISTER(tb_decay_scan_rect)
TB_TAPE_REGISTER(tb_decay_step_f32)
TB_TAPE_REGISTER(tb_decay_step_bf16)
