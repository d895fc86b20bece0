// Gated delta rule: a state S (dk x dv per head, 32-bit, in the request's state slot) whose content for a key is
// corrected towards the token's value instead of being added to,
//
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q,
//
// with one decay g = exp(-exp(a_log) softplus(a + dt_bias)) and one step beta = sigmoid(b) per head and token, k a unit
// vector and q a unit vector times a constant.
//
//   delta_prepare   per token: the short causal convolution of the q, k and v projections with SiLU, the unit norms of q
//                   and k per head, beta and g
//   delta_walk      the recurrence token by token, four columns of the state a thread (steps of few tokens per request:
//                   the state's bytes are what takes the time)
//   delta_coefs, delta_blocks
//                   the recurrence in blocks of eight tokens (long portions: the chain from token to token is what takes the
//                   time). With S the state before the block, a_j = S^T k_j and b_j = S^T q_j are taken for all eight at
//                   once, and the corrections are carried between the tokens by the products of their keys:
//                     u_j = beta_j v_j - beta_j D_j a_j - sum_(i<j) M_ji u_i,     M_ji = beta_j G_ij (k_j . k_i)
//                     o_j = D_j b_j + sum_(i<=j) N_ji u_i,                        N_ji = G_ij (q_j . k_i)
//                     S <- D_7 S + sum_i G_i7 k_i u_i^T,      G_ij = g_(i+1) .. g_j,  D_j = g_0 .. g_j
//                   which is the same recurrence with its sums in another order. delta_coefs prepares the coefficients of
//                   every token (they are common to all columns of a head); blocks are counted from a segment's first row
// Both forms also rewrite the request's last inputs of the convolution (which delta_prepare has finished reading).
//
// A step's rows are segments (one per request: seg_start, seg_len, state_slots as the step's descriptor holds them on the
// device). A token's result depends on its own request only; how the request was cut into steps shows in rounding only.
// Everything is 32-bit.
#include "common.cuh"

namespace gi {

__device__ __forceinline__ float delta_silu(float z) { return z * (1.0f / (1.0f + expf(-z))); }
__device__ __forceinline__ float delta_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

constexpr int kDeltaMaxDim = 256;

struct DeltaArgs {
    const float* proj; int ld, in_off;                    // projections [T, ld]: q, k, v side by side from column in_off
    int b_off, a_off;                                     // columns of b and a (H each)
    const float* conv;                                    // [C, taps], the last column weighs the token itself
    const float* a_log; const float* dt_bias;             // [H]
    float* state; long long slot_stride, state_off, conv_off;      // per slot: [H, dk, dv] at state_off, [taps - 1, C] at conv_off
    const int* row_req; const int* seg_start; const int* seg_len; const int* state_slots;
    float* qkv;                                           // [T, C]: q, k, v as the recurrence takes them
    float* gates;                                         // [T, 2 H]: beta, then g
    float* coefs;                                         // [T, H, kCoefs]: see delta_coefs_kernel (delta_blocks)
    float* out;                                           // [T, H * dv]
    int T, H, G, dk, dv, C, taps;
    float q_scale, unit_eps;
};

// The convolution of one warp's channels (U a lane) over consecutive rows. With TAPS > 0 the weights and the last inputs
// stay in registers and a row costs one load a channel; TAPS 0 takes any number of taps and reads them again per row.
template <int U, int TAPS>
struct ConvRun {
    float w[U][TAPS > 0 ? TAPS : 1], hist[U][TAPS > 1 ? TAPS - 1 : 1];

    __device__ __forceinline__ void start(const DeltaArgs& p, int first, int n, int lane) {
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int u = 0; u < U; ++u) {
#pragma unroll
                for (int j = 0; j < TAPS; ++j)
                    w[u][j] = lane + 32 * u < n ? p.conv[static_cast<size_t>(first + lane + 32 * u) * TAPS + j] : 0.f;
            }
        }
    }
    // the inputs before row t, which is row ``rel`` of its request's rows
    __device__ __forceinline__ void reach_back(const DeltaArgs& p, int t, int rel, const float* st, int first, int n, int lane) {
        if constexpr (TAPS > 1) {
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int c = first + lane + 32 * u;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const int back = TAPS - 1 - j;
                    hist[u][j] = lane + 32 * u >= n ? 0.f
                                 : back <= rel ? p.proj[static_cast<size_t>(t - back) * p.ld + p.in_off + c]
                                               : st[static_cast<size_t>(TAPS - 1 + rel - back) * p.C + c];
                }
            }
        }
    }
    __device__ __forceinline__ void row(const DeltaArgs& p, int t, int rel, const float* st, int first, int n, int lane, float (&y)[U]) {
        if constexpr (TAPS > 0) {
            float x[U];
#pragma unroll
            for (int u = 0; u < U; ++u)
                x[u] = lane + 32 * u < n ? p.proj[static_cast<size_t>(t) * p.ld + p.in_off + first + lane + 32 * u] : 0.f;
#pragma unroll
            for (int u = 0; u < U; ++u) {
                float acc = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(w[u][j], hist[u][j], acc);
                acc = fmaf(w[u][TAPS - 1], x[u], acc);
#pragma unroll
                for (int j = 0; j + 1 < TAPS - 1; ++j) hist[u][j] = hist[u][j + 1];
                if constexpr (TAPS > 1) hist[u][TAPS - 2] = x[u];
                y[u] = delta_silu(acc);
            }
        } else {
#pragma unroll
            for (int u = 0; u < U; ++u) {
                y[u] = 0.f;
                if (lane + 32 * u < n) {
                    const int c = first + lane + 32 * u;
                    float acc = 0.f;
                    for (int j = 0; j < p.taps; ++j) {
                        const int back = p.taps - 1 - j;             // how many tokens before t
                        const float x = back <= rel ? p.proj[static_cast<size_t>(t - back) * p.ld + p.in_off + c]
                                                    : st[static_cast<size_t>(p.taps - 1 + rel - back) * p.C + c];
                        acc = fmaf(p.conv[static_cast<size_t>(c) * p.taps + j], x, acc);
                    }
                    y[u] = delta_silu(acc);
                }
            }
        }
    }
};

// A warp per item and run of consecutive tokens. Items of a token: the q heads, the k heads (convolution, SiLU, unit norm),
// runs of 128 channels of v (convolution, SiLU), and one item for beta and g.
constexpr int kPrepRun = 8;           // tokens of a run (steps of few tokens per request: one)

template <int U, int TAPS>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaArgs p, int run) {
    pdl_prologue();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int item = blockIdx.x * 8 + warp;
    const int n_v = (p.H * p.dv + 127) / 128;
    const int n_items = 2 * p.G + n_v + 1;
    if (item >= n_items) return;
    const int t0 = blockIdx.y * run, t1 = min(p.T, t0 + run);
    if (item == n_items - 1) {
        for (int i = lane; i < (t1 - t0) * p.H; i += 32) {
            const int t = t0 + i / p.H, h = i % p.H;
            const float* row = p.proj + static_cast<size_t>(t) * p.ld;
            p.gates[static_cast<size_t>(t) * 2 * p.H + h] = 1.0f / (1.0f + expf(-row[p.b_off + h]));
            p.gates[static_cast<size_t>(t) * 2 * p.H + p.H + h] = expf(-expf(p.a_log[h]) * delta_softplus(row[p.a_off + h] + p.dt_bias[h]));
        }
        return;
    }
    const bool is_v = item >= 2 * p.G;
    const int first = is_v ? 2 * p.G * p.dk + (item - 2 * p.G) * 128 : item * p.dk;
    const int n = is_v ? min(128, p.C - first) : p.dk;
    ConvRun<U, TAPS> conv;
    conv.start(p, first, n, lane);
    for (int t = t0; t < t1; ++t) {
        const int r = p.row_req[t], rel = t - p.seg_start[r];
        const float* st = p.state + static_cast<long long>(p.state_slots[r]) * p.slot_stride + p.conv_off;
        if (t == t0 || rel == 0) conv.reach_back(p, t, rel, st, first, n, lane);
        float y[U];
        conv.row(p, t, rel, st, first, n, lane, y);
        float f = 1.f;
        if (!is_v) {
            float ss = 0.f;
#pragma unroll
            for (int u = 0; u < U; ++u) ss = fmaf(y[u], y[u], ss);
            f = (item < p.G ? p.q_scale : 1.0f) / sqrtf(warp_sum(ss) + p.unit_eps);
        }
        float* dst = p.qkv + static_cast<size_t>(t) * p.C + first;
#pragma unroll
        for (int u = 0; u < U; ++u)
            if (lane + 32 * u < n) dst[lane + 32 * u] = y[u] * f;
    }
}

// The coefficients of a token for every head (delta_blocks): its place in its block is j = rel % 8. Per (token, head), kCoefs
// floats: M_j0 .. M_j7 (zero from i = j on), N_j0 .. N_j7 (zero behind i = j), beta_j, beta_j D_j, D_j, G_j,last (last: the
// block's last token that exists). A warp per (token, key head); the products are taken once for the heads that share it.
constexpr int kBlock = 8, kCoefs = 20;

template <int U>
__global__ void __launch_bounds__(256)
delta_coefs_kernel(const DeltaArgs p) {
    pdl_prologue();
    __shared__ float s_dot[8][2 * kBlock];                    // per warp: k_j . k_(j-l), then q_j . k_(j-l), by lag l
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = blockIdx.x * 8 + warp, t = blockIdx.y;
    if (g >= p.G) return;
    const int r = p.row_req[t], rel = t - p.seg_start[r];
    const int j = rel % kBlock, last = min(kBlock - 1, j + p.seg_len[r] - 1 - rel);
    const float* row = p.qkv + static_cast<size_t>(t) * p.C;
    float q[U], k[U], kk[kBlock], qk[kBlock];
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int i = lane + 32 * u;
        q[u] = i < p.dk ? row[g * p.dk + i] : 0.f;
        k[u] = i < p.dk ? row[(p.G + g) * p.dk + i] : 0.f;
    }
#pragma unroll
    for (int l = 0; l < kBlock; ++l) {
        kk[l] = qk[l] = 0.f;
        if (l <= j) {
            const float* back = p.qkv + static_cast<size_t>(t - l) * p.C + (p.G + g) * p.dk;
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int i = lane + 32 * u;
                const float x = l == 0 ? k[u] : i < p.dk ? back[i] : 0.f;
                kk[l] = fmaf(k[u], x, kk[l]);
                qk[l] = fmaf(q[u], x, qk[l]);
            }
        }
    }
#pragma unroll
    for (int l = 0; l < kBlock; ++l) {
        if (l <= j) {
            kk[l] = warp_sum(kk[l]);
            qk[l] = warp_sum(qk[l]);
        }
    }
    if (lane == 0) {
#pragma unroll
        for (int l = 0; l < kBlock; ++l) { s_dot[warp][l] = kk[l]; s_dot[warp][kBlock + l] = qk[l]; }
    }
    __syncwarp();
    // a lane per (head that shares the key head, column of the coefficients)
    const int share = p.H / p.G;
    for (int e = lane; e < share * kBlock; e += 32) {
        const int h = g * share + e / kBlock, i = e % kBlock;
        const float* gb = p.gates + static_cast<size_t>(t) * 2 * p.H + h;            // row t: beta, then g behind H floats
        const long long stride = 2 * p.H;
        float* out = p.coefs + (static_cast<size_t>(t) * p.H + h) * kCoefs;
        const float beta = gb[0];
        float G = 1.f;                                                               // G_ij
        for (int b = 0; b < j - i; ++b) G *= gb[p.H - b * stride];
        out[i] = i < j ? beta * G * s_dot[warp][j - i] : 0.f;
        out[kBlock + i] = i <= j ? G * s_dot[warp][kBlock + j - i] : 0.f;
        if (i == 0) {
            const float D = G * gb[p.H - j * stride];
            float F = 1.f;
            for (int b = 1; b <= last - j; ++b) F *= gb[p.H + b * stride];
            out[2 * kBlock] = beta;
            out[2 * kBlock + 1] = beta * D;
            out[2 * kBlock + 2] = D;
            out[2 * kBlock + 3] = F;
        }
    }
}

__device__ __forceinline__ void delta_cp_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}
__device__ __forceinline__ void delta_cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}

// The convolution's last taps - 1 inputs of a request, a run of channels per block of the (columns, heads) grid.
__device__ __forceinline__ void keep_conv_inputs(const DeltaArgs& p, float* slot, int n, int s0, int tid, int threads) {
    const int keep = p.taps - 1;
    if (keep <= 0) return;
    float* st = slot + p.conv_off;
    const int blocks = gridDim.x * gridDim.y, b = blockIdx.y * gridDim.x + blockIdx.x;
    const int run = (p.C + blocks - 1) / blocks;
    for (int c = b * run + tid; c < min(p.C, (b + 1) * run); c += threads) {
        float vals[16];
        for (int j = 0; j < keep; ++j) {
            const int rel = n - keep + j;                 // index among the segment's rows; negative: an older input
            vals[j] = rel >= 0 ? p.proj[static_cast<size_t>(s0 + rel) * p.ld + p.in_off + c] : st[static_cast<size_t>(keep + rel) * p.C + c];
        }
        for (int j = 0; j < keep; ++j) st[static_cast<size_t>(j) * p.C + c] = vals[j];
    }
}

constexpr int kDeltaWarps = 4;
constexpr int kDeltaThreads = kDeltaWarps * 32;

// What both forms stage per token: q, k, the block's columns of v, and beta and g or the coefficients.
template <int kDk, int kCols, int kChunk, bool kBlocks>
struct DeltaStage {
    float k[kChunk][kDk], q[kChunk][kDk], v[kChunk][kCols];
    float c[kBlocks ? kChunk : 1][kCoefs];
    float b[kChunk], g[kChunk];

    // rows c0 .. of a segment that starts at row s0; tokens beyond its n rows are left as they are (delta_blocks: neutral)
    __device__ __forceinline__ void request(const DeltaArgs& p, int s0, int n, int c0, int h, int hq, int col0, int n_cols, int wide, int tid) {
        const int m = min(kChunk, n - c0);
        const float* base = p.qkv + static_cast<size_t>(s0 + c0) * p.C;
        const int k_off = p.G * p.dk, v_off = 2 * p.G * p.dk + h * p.dv + col0;
        if (wide) {                                                     // heads in whole 16-byte pieces
            const int q4 = p.dk / 4, v4 = n_cols / 4;
            // a warp per row, so that no thread divides by the row length
            for (int tt = tid >> 5; tt < m; tt += kDeltaWarps) {
                const float* row = base + static_cast<size_t>(tt) * p.C + hq * p.dk;
                for (int i = tid & 31; i < q4; i += 32) {
                    delta_cp_async16(&q[tt][4 * i], row + 4 * i);
                    delta_cp_async16(&k[tt][4 * i], row + k_off + 4 * i);
                }
                const float* vr = base + static_cast<size_t>(tt) * p.C + v_off;
                for (int i = tid & 31; i < v4; i += 32) delta_cp_async16(&v[tt][4 * i], vr + 4 * i);
            }
        } else {
            for (int tt = tid >> 5; tt < m; tt += kDeltaWarps) {
                const float* row = base + static_cast<size_t>(tt) * p.C + hq * p.dk;
                for (int i = tid & 31; i < p.dk; i += 32) {
                    delta_cp_async4(&q[tt][i], row + i);
                    delta_cp_async4(&k[tt][i], row + k_off + i);
                }
                const float* vr = base + static_cast<size_t>(tt) * p.C + v_off;
                for (int i = tid & 31; i < n_cols; i += 32) delta_cp_async4(&v[tt][i], vr + i);
            }
        }
        if (kBlocks) {
            if (tid < m * (kCoefs / 4)) {
                const int tt = tid / (kCoefs / 4), i = tid % (kCoefs / 4) * 4;
                delta_cp_async16(&c[kBlocks ? tt : 0][i], p.coefs + (static_cast<size_t>(s0 + c0 + tt) * p.H + h) * kCoefs + i);
            }
        } else if (tid < m) {
            const float* gr = p.gates + static_cast<size_t>(s0 + c0 + tid) * 2 * p.H + h;
            delta_cp_async4(&b[tid], gr);
            delta_cp_async4(&g[tid], gr + p.H);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
};

// Eight lanes share a column: lane group member rg holds the rows 4 (8 i + rg) .. + 3 (i < RPT / 4) of four columns in
// registers, and a sum over the rows needs one exchange over the eight lanes.
constexpr int kDeltaGroup = 8;

template <int RPT>
__global__ void __launch_bounds__(kDeltaThreads)
delta_walk_kernel(const DeltaArgs p, int wide) {
    constexpr int CPT = 4;
    constexpr int kDk = RPT * kDeltaGroup;
    constexpr int kCols = kDeltaWarps * (32 / kDeltaGroup) * CPT;       // columns of a block
    constexpr int kChunk = kDk > 128 ? 4 : 8;                           // tokens staged at a time
    __shared__ __align__(16) DeltaStage<kDk, kCols, kChunk, false> stg[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, r = blockIdx.z;
    const int hq = h / (p.H / p.G);
    const int col0 = blockIdx.x * kCols;
    const int rg = lane % kDeltaGroup;
    const int my = (warp * (32 / kDeltaGroup) + lane / kDeltaGroup) * CPT;      // this thread's first column in the block
    // the padding rows of k and q stay zero
    for (int e = tid; e < 2 * kChunk * (kDk - p.dk); e += kDeltaThreads) {
        const int pad = kDk - p.dk, s = e / pad / kChunk, tt = e / pad % kChunk, i = p.dk + e % pad;
        stg[s].k[tt][i] = 0.f;
        stg[s].q[tt][i] = 0.f;
    }
    pdl_prologue();
    const int n = p.seg_len[r], s0 = p.seg_start[r];
    float* slot = p.state + static_cast<long long>(p.state_slots[r]) * p.slot_stride;
    float* S = slot + p.state_off + static_cast<size_t>(h) * p.dk * p.dv;
    const int n_cols = min(kCols, p.dv - col0);
    stg[0].request(p, s0, n, 0, h, hq, col0, n_cols, wide, tid);

    float s[RPT][CPT];
    const bool vec = p.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(S) & 15) == 0;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int row = (i / 4 * kDeltaGroup + rg) * 4 + i % 4;
        const float* src = S + static_cast<size_t>(row) * p.dv + col0 + my;
        if (vec) {
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (row < p.dk && my < n_cols) x = *reinterpret_cast<const float4*>(src);
            s[i][0] = x.x; s[i][1] = x.y; s[i][2] = x.z; s[i][3] = x.w;
        } else {
#pragma unroll
            for (int c = 0; c < CPT; ++c) s[i][c] = (row < p.dk && my + c < n_cols) ? src[c] : 0.f;
        }
    }
    for (int c0 = 0, st = 0; c0 < n; c0 += kChunk, st ^= 1) {
        const int m = min(kChunk, n - c0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                   // the chunk is there, and everyone is done with the other stage
        if (c0 + kChunk < n) stg[st ^ 1].request(p, s0, n, c0 + kChunk, h, hq, col0, n_cols, wide, tid);
        for (int tt = 0; tt < m; ++tt) {
            const float g = stg[st].g[tt], beta = stg[st].b[tt];
            const float4* k4 = reinterpret_cast<const float4*>(&stg[st].k[tt][rg * 4]);
            const float4* q4 = reinterpret_cast<const float4*>(&stg[st].q[tt][rg * 4]);
            float dot[CPT], o[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) dot[c] = o[c] = 0.f;
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
                const float4 kk = k4[i4 * kDeltaGroup];
                const float kr[4] = {kk.x, kk.y, kk.z, kk.w};
#pragma unroll
                for (int u = 0; u < 4; ++u) {
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        s[4 * i4 + u][c] *= g;
                        dot[c] = fmaf(kr[u], s[4 * i4 + u][c], dot[c]);
                    }
                }
            }
#pragma unroll
            for (int x = 1; x < kDeltaGroup; x <<= 1) {
#pragma unroll
                for (int c = 0; c < CPT; ++c) dot[c] += __shfl_xor_sync(0xffffffffu, dot[c], x);
            }
            float u_[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) u_[c] = beta * (stg[st].v[tt][my + c] - dot[c]);
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
                const float4 kk = k4[i4 * kDeltaGroup], qq = q4[i4 * kDeltaGroup];
                const float kr[4] = {kk.x, kk.y, kk.z, kk.w}, qr[4] = {qq.x, qq.y, qq.z, qq.w};
#pragma unroll
                for (int u = 0; u < 4; ++u) {
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        s[4 * i4 + u][c] = fmaf(kr[u], u_[c], s[4 * i4 + u][c]);
                        o[c] = fmaf(qr[u], s[4 * i4 + u][c], o[c]);
                    }
                }
            }
#pragma unroll
            for (int x = 1; x < kDeltaGroup; x <<= 1) {
#pragma unroll
                for (int c = 0; c < CPT; ++c) o[c] += __shfl_xor_sync(0xffffffffu, o[c], x);
            }
            if (rg == 0) {
                float* dst = p.out + static_cast<size_t>(s0 + c0 + tt) * p.H * p.dv + static_cast<size_t>(h) * p.dv + col0 + my;
#pragma unroll
                for (int c = 0; c < CPT; ++c)
                    if (my + c < n_cols) dst[c] = o[c];
            }
        }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int row = (i / 4 * kDeltaGroup + rg) * 4 + i % 4;
        float* dst = S + static_cast<size_t>(row) * p.dv + col0 + my;
        if (vec) {
            if (row < p.dk && my < n_cols) *reinterpret_cast<float4*>(dst) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
        } else {
#pragma unroll
            for (int c = 0; c < CPT; ++c)
                if (row < p.dk && my + c < n_cols) dst[c] = s[i][c];
        }
    }
    keep_conv_inputs(p, slot, n, s0, tid, kDeltaThreads);
}

// Eight tokens at a time. Sixteen lanes share two columns of the state: lane group member rg holds the rows
// 4 (16 i + rg) .. + 3 (i < RPT / 4). The 32 sums over the rows (a_j and b_j of two columns) are spread over the lanes in two
// halving exchanges (bit 3 of rg keeps a column, bit 2 keeps a or b) and completed in two more; the lanes that hold a column's
// a_j solve for its u_j, everyone gets both columns' u_j, and the lanes that hold b_j read out.
constexpr int kWideGroup = 16;

template <int RPT>
__global__ void __launch_bounds__(kDeltaThreads)
delta_blocks_kernel(const DeltaArgs p, int wide) {
    constexpr int kDk = RPT * kWideGroup;
    constexpr int kCols = kDeltaWarps * (32 / kWideGroup) * 2;          // columns of a block
    constexpr int kChunk = kDk > 128 ? 8 : 16;                          // tokens staged at a time
    __shared__ __align__(16) DeltaStage<kDk, kCols, kChunk, true> stg[2];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, r = blockIdx.z;
    const int hq = h / (p.H / p.G);
    const int col0 = blockIdx.x * kCols;
    const int rg = lane % kWideGroup;
    const int my = (warp * (32 / kWideGroup) + lane / kWideGroup) * 2;  // the first of this thread's two columns in the block
    const int c_mine = (rg >> 3) & 1;                                   // the column whose sums end up with this lane,
    const bool reads = (rg >> 2) & 1;                                   // and which: b_j (else a_j)
    // rows beyond dk, columns beyond dv and tokens beyond the segment's end are neutral: all zero
    for (int e = tid; e < static_cast<int>(sizeof(stg) / 4); e += kDeltaThreads) reinterpret_cast<float*>(stg)[e] = 0.f;
    pdl_prologue();
    __syncthreads();
    const int n = p.seg_len[r], s0 = p.seg_start[r];
    float* slot = p.state + static_cast<long long>(p.state_slots[r]) * p.slot_stride;
    float* S = slot + p.state_off + static_cast<size_t>(h) * p.dk * p.dv;
    const int n_cols = min(kCols, p.dv - col0);
    stg[0].request(p, s0, n, 0, h, hq, col0, n_cols, wide, tid);
    float s[RPT][2];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int row = (i / 4 * kWideGroup + rg) * 4 + i % 4;
#pragma unroll
        for (int c = 0; c < 2; ++c) s[i][c] = (row < p.dk && my + c < n_cols) ? S[static_cast<size_t>(row) * p.dv + col0 + my + c] : 0.f;
    }
    float* out = p.out + static_cast<size_t>(s0) * p.H * p.dv + static_cast<size_t>(h) * p.dv + col0 + my + c_mine;
    const bool emits = reads && my + c_mine < n_cols;
    for (int c0 = 0, st = 0; c0 < n; c0 += kChunk, st ^= 1) {
        const int m = min(kChunk, n - c0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                   // the chunk is there, and everyone is done with the other stage
        if (c0 + kChunk < n) stg[st ^ 1].request(p, s0, n, c0 + kChunk, h, hq, col0, n_cols, wide, tid);
        if (m % kBlock) {                                  // the last block is not whole: its missing tokens (whose places may
            for (int e = tid; e < (kBlock - m % kBlock) * kCoefs; e += kDeltaThreads)       // hold an earlier chunk's) do nothing
                stg[st].c[m + e / kCoefs][e % kCoefs] = 0.f;
            __syncthreads();
        }
        const auto& x = stg[st];
        for (int tt = 0; tt < m; tt += kBlock) {
            float a[2][kBlock], b[2][kBlock];
            float4 kr[kBlock][RPT / 4];
#pragma unroll
            for (int j = 0; j < kBlock; ++j) a[0][j] = a[1][j] = b[0][j] = b[1][j] = 0.f;
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
#pragma unroll
                for (int j = 0; j < kBlock; ++j) {
                    const float4 kk = *reinterpret_cast<const float4*>(&x.k[tt + j][(i4 * kWideGroup + rg) * 4]);
                    const float4 qq = *reinterpret_cast<const float4*>(&x.q[tt + j][(i4 * kWideGroup + rg) * 4]);
                    kr[j][i4] = kk;
#pragma unroll
                    for (int c = 0; c < 2; ++c) {
                        a[c][j] = fmaf(kk.x, s[4 * i4][c], a[c][j]);         b[c][j] = fmaf(qq.x, s[4 * i4][c], b[c][j]);
                        a[c][j] = fmaf(kk.y, s[4 * i4 + 1][c], a[c][j]);     b[c][j] = fmaf(qq.y, s[4 * i4 + 1][c], b[c][j]);
                        a[c][j] = fmaf(kk.z, s[4 * i4 + 2][c], a[c][j]);     b[c][j] = fmaf(qq.z, s[4 * i4 + 2][c], b[c][j]);
                        a[c][j] = fmaf(kk.w, s[4 * i4 + 3][c], a[c][j]);     b[c][j] = fmaf(qq.w, s[4 * i4 + 3][c], b[c][j]);
                    }
                }
            }
            float w[kBlock];                               // this lane's sums: a_j or b_j of column c_mine
#pragma unroll
            for (int j = 0; j < kBlock; ++j) {
                // bit 3 keeps a column, bit 2 keeps a or b
                const float ka = c_mine ? a[1][j] : a[0][j], sa = c_mine ? a[0][j] : a[1][j];
                const float kb = c_mine ? b[1][j] : b[0][j], sb = c_mine ? b[0][j] : b[1][j];
                const float ta = ka + __shfl_xor_sync(0xffffffffu, sa, 8);
                const float tb = kb + __shfl_xor_sync(0xffffffffu, sb, 8);
                w[j] = (reads ? tb : ta) + __shfl_xor_sync(0xffffffffu, reads ? ta : tb, 4);
            }
#pragma unroll
            for (int o = 2; o > 0; o >>= 1) {
#pragma unroll
                for (int j = 0; j < kBlock; ++j) w[j] += __shfl_xor_sync(0xffffffffu, w[j], o);
            }
            // u_j of column c_mine on the lanes that hold a_j
            float u[kBlock];
#pragma unroll
            for (int j = 0; j < kBlock; ++j) {
                const float4 e = *reinterpret_cast<const float4*>(&x.c[tt + j][2 * kBlock]);           // beta, beta D, D, G_j,last
                float acc = fmaf(e.x, x.v[tt + j][my + c_mine], -e.y * w[j]);
                const float4 m0 = *reinterpret_cast<const float4*>(&x.c[tt + j][0]), m1 = *reinterpret_cast<const float4*>(&x.c[tt + j][4]);
                const float mm[kBlock] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
#pragma unroll
                for (int i = 0; i < j; ++i) acc = fmaf(-mm[i], u[i], acc);
                u[j] = acc;
            }
            float u0[kBlock], u1[kBlock];                  // both columns' on every lane
            const int src = lane & kWideGroup;
#pragma unroll
            for (int j = 0; j < kBlock; ++j) {
                u0[j] = __shfl_sync(0xffffffffu, u[j], src);
                u1[j] = __shfl_sync(0xffffffffu, u[j], src + 8);
            }
            float o_even = 0.f, o_odd = 0.f;               // the read-outs of tokens 2 (rg & 3) and 2 (rg & 3) + 1
#pragma unroll
            for (int j = 0; j < kBlock; ++j) {
                const float4 n0 = *reinterpret_cast<const float4*>(&x.c[tt + j][kBlock]), n1 = *reinterpret_cast<const float4*>(&x.c[tt + j][kBlock + 4]);
                const float nn[kBlock] = {n0.x, n0.y, n0.z, n0.w, n1.x, n1.y, n1.z, n1.w};
                float o = x.c[tt + j][2 * kBlock + 2] * w[j];
#pragma unroll
                for (int i = 0; i <= j; ++i) o = fmaf(nn[i], c_mine ? u1[i] : u0[i], o);
                if ((rg & 3) == j / 2) { if (j & 1) o_odd = o; else o_even = o; }
            }
            const int te = c0 + tt + 2 * (rg & 3);
            if (emits && te < n) out[static_cast<size_t>(te) * p.H * p.dv] = o_even;
            if (emits && te + 1 < n) out[static_cast<size_t>(te + 1) * p.H * p.dv] = o_odd;
            // the state after the block
            const float d = x.c[tt + min(kBlock, m - tt) - 1][2 * kBlock + 2];
#pragma unroll
            for (int j = 0; j < kBlock; ++j) {
                const float f = x.c[tt + j][2 * kBlock + 3];
                u0[j] *= f;
                u1[j] *= f;
            }
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
#pragma unroll
                for (int e = 0; e < 4; ++e) { s[4 * i4 + e][0] *= d; s[4 * i4 + e][1] *= d; }
#pragma unroll
                for (int j = 0; j < kBlock; ++j) {
                    const float4 kk = kr[j][i4];
                    s[4 * i4][0] = fmaf(kk.x, u0[j], s[4 * i4][0]);         s[4 * i4][1] = fmaf(kk.x, u1[j], s[4 * i4][1]);
                    s[4 * i4 + 1][0] = fmaf(kk.y, u0[j], s[4 * i4 + 1][0]); s[4 * i4 + 1][1] = fmaf(kk.y, u1[j], s[4 * i4 + 1][1]);
                    s[4 * i4 + 2][0] = fmaf(kk.z, u0[j], s[4 * i4 + 2][0]); s[4 * i4 + 2][1] = fmaf(kk.z, u1[j], s[4 * i4 + 2][1]);
                    s[4 * i4 + 3][0] = fmaf(kk.w, u0[j], s[4 * i4 + 3][0]); s[4 * i4 + 3][1] = fmaf(kk.w, u1[j], s[4 * i4 + 3][1]);
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int row = (i / 4 * kWideGroup + rg) * 4 + i % 4;
#pragma unroll
        for (int c = 0; c < 2; ++c)
            if (row < p.dk && my + c < n_cols) S[static_cast<size_t>(row) * p.dv + col0 + my + c] = s[i][c];
    }
    keep_conv_inputs(p, slot, n, s0, tid, kDeltaThreads);
}

template <int RPT>
static void launch_delta_walk(const DeltaArgs& a, int R, int wide, cudaStream_t st) {
    constexpr unsigned cols = kDeltaWarps * (32 / kDeltaGroup) * 4;
    launch_kernel((delta_walk_kernel<RPT>), dim3((a.dv + cols - 1) / cols, a.H, R), dim3(kDeltaThreads), 0, st, a, wide);
}

template <int RPT>
static void launch_delta_blocks(const DeltaArgs& a, int R, int wide, cudaStream_t st) {
    constexpr unsigned cols = kDeltaWarps * (32 / kWideGroup) * 2;
    launch_kernel_as(false, (delta_blocks_kernel<RPT>), dim3((a.dv + cols - 1) / cols, a.H, R), dim3(kDeltaThreads), 0, st, a, wide);
}

template <int U>
static void launch_delta_prepare(const DeltaArgs& a, int run, cudaStream_t st) {
    const int items = 2 * a.G + (a.H * a.dv + 127) / 128 + 1;
    const dim3 grid((items + 7) / 8, (a.T + run - 1) / run);
    switch (a.taps) {
        case 1: launch_kernel((delta_prepare_kernel<U, 1>), grid, dim3(256), 0, st, a, run); break;
        case 2: launch_kernel((delta_prepare_kernel<U, 2>), grid, dim3(256), 0, st, a, run); break;
        case 3: launch_kernel((delta_prepare_kernel<U, 3>), grid, dim3(256), 0, st, a, run); break;
        case 4: launch_kernel((delta_prepare_kernel<U, 4>), grid, dim3(256), 0, st, a, run); break;
        default: launch_kernel((delta_prepare_kernel<U, 0>), grid, dim3(256), 0, st, a, run); break;
    }
}

}  // namespace gi

using namespace gi;

extern "C" int gi_gated_delta_coefs() { return kCoefs; }

// delta_prepare, then the recurrence: with the workspace ``coefs`` in blocks of eight tokens (long portions), without it token
// by token (steps of few tokens per request).
static int gi_gated_delta_impl(const float* proj, int ld, int in_off, int b_off, int a_off, const float* conv, int taps,
                               const float* a_log, const float* dt_bias, float q_scale, float unit_eps, float* state,
                               long long slot_stride, long long state_off, long long conv_off, const int* row_req,
                               const int* seg_start, const int* seg_len, const int* state_slots, float* qkv, float* gates,
                               float* coefs, float* out, int T, int R, int H, int G, int dk, int dv, void* stream) {
    if (T == 0 || R == 0) return 0;
    GI_REQUIRE(T > 0 && R > 0 && H > 0 && G > 0 && dk > 0 && dv > 0, "gated_delta: sizes must be positive");
    GI_REQUIRE(H % G == 0, "gated_delta: %d heads are not a multiple of %d key heads", H, G);
    GI_REQUIRE(dk <= kDeltaMaxDim, "gated_delta: %d state rows per head exceed %d", dk, kDeltaMaxDim);
    GI_REQUIRE(taps >= 1 && taps <= 17, "gated_delta: %d convolution taps are not supported (1 to 17)", taps);
    const int C = 2 * G * dk + H * dv;
    GI_REQUIRE(in_off >= 0 && in_off + C <= ld && b_off >= 0 && b_off + H <= ld && a_off >= 0 && a_off + H <= ld,
               "gated_delta: the columns lie outside the input row of %d", ld);
    GI_REQUIRE(reinterpret_cast<uintptr_t>(coefs) % 16 == 0, "gated_delta: the workspace of coefficients must be 16-byte aligned");
    const bool blocks = coefs != nullptr;
    const int run = blocks ? kPrepRun : 1;
    GI_REQUIRE(H <= 65535 && R <= 65535 && T <= 65535, "gated_delta: the grid limit 65535 is exceeded");
    DeltaArgs a{proj, ld, in_off, b_off, a_off, conv, a_log, dt_bias, state, slot_stride, state_off, conv_off, row_req, seg_start,
                seg_len, state_slots, qkv, gates, coefs, out, T, H, G, dk, dv, C, taps, q_scale, unit_eps};
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (dk <= 128) launch_delta_prepare<4>(a, run, st);
    else launch_delta_prepare<8>(a, run, st);
    if (check_launch("gated_delta (prepare)")) return 1;
    const int wide = dk % 4 == 0 && dv % 4 == 0 && reinterpret_cast<uintptr_t>(qkv) % 16 == 0;
    if (blocks) {
        const dim3 grid((G + 7) / 8, T);
        if (dk <= 128) launch_kernel((delta_coefs_kernel<4>), grid, dim3(256), 0, st, a);
        else launch_kernel((delta_coefs_kernel<8>), grid, dim3(256), 0, st, a);
        if (check_launch("gated_delta (coefficients)")) return 1;
        if (dk <= 64) launch_delta_blocks<4>(a, R, wide, st);
        else if (dk <= 128) launch_delta_blocks<8>(a, R, wide, st);
        else if (dk <= 192) launch_delta_blocks<12>(a, R, wide, st);
        else launch_delta_blocks<16>(a, R, wide, st);
        return check_launch("gated_delta (blocks)");
    }
    if (dk <= 32) launch_delta_walk<4>(a, R, wide, st);
    else if (dk <= 64) launch_delta_walk<8>(a, R, wide, st);
    else if (dk <= 96) launch_delta_walk<12>(a, R, wide, st);
    else if (dk <= 128) launch_delta_walk<16>(a, R, wide, st);
    else if (dk <= 192) launch_delta_walk<24>(a, R, wide, st);
    else launch_delta_walk<32>(a, R, wide, st);
    return check_launch("gated_delta");
}

extern "C" int gi_gated_delta(const float* proj, int ld, int in_off, int b_off, int a_off, const float* conv, int taps, const float* a_log, const float* dt_bias, float q_scale, float unit_eps, float* state, long long slot_stride, long long state_off, long long conv_off, const int* row_req, const int* seg_start, const int* seg_len, const int* state_slots, float* qkv, float* gates, float* coefs, float* out, int T, int R, int H, int G, int dk, int dv, void* stream) {
    return gi::dispatch(gi_gated_delta_impl, proj, ld, in_off, b_off, a_off, conv, taps, a_log, dt_bias, q_scale, unit_eps, state, slot_stride, state_off, conv_off, row_req, seg_start, seg_len, state_slots, qkv, gates, coefs, out, T, R, H, G, dk, dv, stream);
}
