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
//   delta_scan      the recurrence over each request's rows in order; its blocks also rewrite the request's last inputs of
//                   the convolution (which delta_prepare has finished reading)
//
// A step's rows are segments (one per request: seg_start, seg_len, state_slots as the step's descriptor holds them on the
// device). Tokens of a segment are taken one after the other with the same arithmetic however the request was cut into
// steps and whatever else is in the batch: an output does not depend on the cut at all, not even by rounding. Everything is
// 32-bit.
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
    float* out;                                           // [T, H * dv]
    int T, H, G, dk, dv, C, taps;
    float q_scale, unit_eps;
};

// A warp per item and kPrepTokens consecutive tokens. Items of a token: the q heads, the k heads (convolution, SiLU, unit
// norm), runs of 128 channels of v (convolution, SiLU), and one item for beta and g.
constexpr int kPrepTokens = 4;

__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaArgs p) {
    pdl_prologue();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int item = blockIdx.x * 8 + warp;
    const int n_v = (p.H * p.dv + 127) / 128;
    const int n_items = 2 * p.G + n_v + 1;
    if (item >= n_items) return;
    const int t0 = blockIdx.y * kPrepTokens, t1 = min(p.T, t0 + kPrepTokens);
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
    const int first = is_v ? 2 * p.G * p.dk + (item - 2 * p.G) * 128 : item * p.dk;      // channel
    const int n = is_v ? min(128, p.C - first) : p.dk;
    for (int t = t0; t < t1; ++t) {
        const int r = p.row_req[t];
        const int rel = t - p.seg_start[r];
        const float* st = p.state + static_cast<long long>(p.state_slots[r]) * p.slot_stride + p.conv_off;
        float v[kDeltaMaxDim / 32];
        float ss = 0.f;
#pragma unroll
        for (int u = 0; u < kDeltaMaxDim / 32; ++u) {
            const int i = lane + 32 * u;
            v[u] = 0.f;
            if (i < n) {
                const int c = first + i;
                const float* w = p.conv + static_cast<size_t>(c) * p.taps;
                float acc = 0.f;
                for (int j = 0; j < p.taps; ++j) {
                    const int back = p.taps - 1 - j;             // how many tokens before t
                    const float x = back <= rel ? p.proj[static_cast<size_t>(t - back) * p.ld + p.in_off + c]
                                                : st[static_cast<size_t>(p.taps - 1 + rel - back) * p.C + c];
                    acc = fmaf(w[j], x, acc);
                }
                v[u] = delta_silu(acc);
                ss = fmaf(v[u], v[u], ss);
            }
        }
        float f = 1.f;
        if (!is_v) {
            ss = warp_sum(ss);
            f = 1.0f / sqrtf(ss + p.unit_eps);
            if (item < p.G) f *= p.q_scale;
        }
        float* dst = p.qkv + static_cast<size_t>(t) * p.C + first;
#pragma unroll
        for (int u = 0; u < kDeltaMaxDim / 32; ++u)
            if (lane + 32 * u < n) dst[lane + 32 * u] = v[u] * f;
    }
}

__device__ __forceinline__ void delta_cp_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}
__device__ __forceinline__ void delta_cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}

// Eight lanes share a column: lane group member rg holds the rows 4 (8 i + rg) .. + 3 (i < RPT / 4) of CPT columns in
// registers, so a token costs 4 operations per state element, and S^T k needs one exchange over the eight lanes. The
// read-out of a token is exchanged together with the next token's S^T k. CPT 1 spreads a head over many warps (long
// portions: the walk over the tokens is what takes the time), CPT 4 reads and writes whole sectors of the state (decoding:
// the state's bytes are what takes the time); an element's arithmetic is the same in both.
constexpr int kDeltaWarps = 4;
constexpr int kDeltaGroup = 8;

template <int RPT, int CPT>
__global__ void __launch_bounds__(kDeltaWarps * 32)
delta_scan_kernel(const DeltaArgs p, int wide) {
    constexpr int kDk = RPT * kDeltaGroup;
    constexpr int kCols = kDeltaWarps * (32 / kDeltaGroup) * CPT;       // columns of a block
    constexpr int kChunk = kDk > 128 ? 8 : 16;                          // tokens staged at a time
    __shared__ __align__(16) float s_k[2][kChunk][kDk];
    __shared__ __align__(16) float s_q[2][kChunk][kDk];
    __shared__ __align__(16) float s_v[2][kChunk][kCols];
    __shared__ float s_b[2][kChunk], s_g[2][kChunk];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, r = blockIdx.z;
    const int hq = h / (p.H / p.G);
    const int col0 = blockIdx.x * kCols;
    const int rg = lane % kDeltaGroup;
    const int my = (warp * (32 / kDeltaGroup) + lane / kDeltaGroup) * CPT;      // this thread's first column in the block
    // the padding rows of k and q stay zero
    if (p.dk < kDk) {
        const int pad = kDk - p.dk;
        for (int e = tid; e < 2 * kChunk * pad; e += kDeltaWarps * 32) {
            s_k[e / pad / kChunk][e / pad % kChunk][p.dk + e % pad] = 0.f;
            s_q[e / pad / kChunk][e / pad % kChunk][p.dk + e % pad] = 0.f;
        }
    }
    pdl_prologue();
    const int n = p.seg_len[r], s0 = p.seg_start[r];
    float* slot = p.state + static_cast<long long>(p.state_slots[r]) * p.slot_stride;
    float* S = slot + p.state_off + static_cast<size_t>(h) * p.dk * p.dv;

    const int n_cols = min(kCols, p.dv - col0);
    auto request = [&](int c0, int stage) {
        const int m = min(kChunk, n - c0);
        const float* base = p.qkv + static_cast<size_t>(s0 + c0) * p.C;
        if (wide) {                                                     // heads in whole 16-byte pieces
            const int q4 = p.dk / 4, v4 = n_cols / 4;
            for (int e = tid; e < m * q4; e += kDeltaWarps * 32) {
                const int tt = e / q4, i = e % q4 * 4;
                const float* row = base + static_cast<size_t>(tt) * p.C + hq * p.dk + i;
                delta_cp_async16(&s_q[stage][tt][i], row);
                delta_cp_async16(&s_k[stage][tt][i], row + p.G * p.dk);
            }
            for (int e = tid; e < m * v4; e += kDeltaWarps * 32)
                delta_cp_async16(&s_v[stage][e / v4][e % v4 * 4], base + static_cast<size_t>(e / v4) * p.C + 2 * p.G * p.dk + h * p.dv + col0 + e % v4 * 4);
        } else {
            for (int e = tid; e < m * p.dk; e += kDeltaWarps * 32) {
                const int tt = e / p.dk, i = e % p.dk;
                const float* row = base + static_cast<size_t>(tt) * p.C + hq * p.dk + i;
                delta_cp_async4(&s_q[stage][tt][i], row);
                delta_cp_async4(&s_k[stage][tt][i], row + p.G * p.dk);
            }
            for (int e = tid; e < m * n_cols; e += kDeltaWarps * 32)
                delta_cp_async4(&s_v[stage][e / n_cols][e % n_cols], base + static_cast<size_t>(e / n_cols) * p.C + 2 * p.G * p.dk + h * p.dv + col0 + e % n_cols);
        }
        if (tid < m) {
            const float* gr = p.gates + static_cast<size_t>(s0 + c0 + tid) * 2 * p.H + h;
            delta_cp_async4(&s_b[stage][tid], gr);
            delta_cp_async4(&s_g[stage][tid], gr + p.H);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    request(0, 0);

    float s[RPT][CPT];
    const bool vec = CPT == 4 && p.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(S) & 15) == 0;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int row = (i / 4 * kDeltaGroup + rg) * 4 + i % 4;
        const float* src = S + static_cast<size_t>(row) * p.dv + col0 + my;
        if (CPT == 4 && vec) {
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (row < p.dk && my < n_cols) x = *reinterpret_cast<const float4*>(src);
            s[i][0] = x.x; s[i][CPT > 1 ? 1 : 0] = CPT > 1 ? x.y : x.x; s[i][CPT > 2 ? 2 : 0] = CPT > 2 ? x.z : x.x; s[i][CPT > 3 ? 3 : 0] = CPT > 3 ? x.w : x.x;
        } else {
#pragma unroll
            for (int c = 0; c < CPT; ++c) s[i][c] = (row < p.dk && my + c < n_cols) ? src[c] : 0.f;
        }
    }

    float o_part[CPT];                 // the read-out of the token before, this lane's rows
#pragma unroll
    for (int c = 0; c < CPT; ++c) o_part[c] = 0.f;
    auto emit = [&](int t, const float (&o)[CPT]) {
        if (rg != 0) return;
        float* dst = p.out + static_cast<size_t>(t) * p.H * p.dv + static_cast<size_t>(h) * p.dv + col0 + my;
#pragma unroll
        for (int c = 0; c < CPT; ++c)
            if (my + c < n_cols) dst[c] = o[c];
    };
    for (int c0 = 0, stage = 0; c0 < n; c0 += kChunk, stage ^= 1) {
        const int m = min(kChunk, n - c0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                   // the chunk is there, and everyone is done with the other stage
        if (c0 + kChunk < n) request(c0 + kChunk, stage ^ 1);
        for (int tt = 0; tt < m; ++tt) {
            const float g = s_g[stage][tt], beta = s_b[stage][tt];
            const float4* k4 = reinterpret_cast<const float4*>(&s_k[stage][tt][rg * 4]);
            const float4* q4 = reinterpret_cast<const float4*>(&s_q[stage][tt][rg * 4]);
            float d[4][CPT];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
#pragma unroll
                for (int c = 0; c < CPT; ++c) d[u][c] = 0.f;
            }
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
                const float4 kk = k4[i4 * kDeltaGroup];
                const float kr[4] = {kk.x, kk.y, kk.z, kk.w};
#pragma unroll
                for (int u = 0; u < 4; ++u) {
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        s[4 * i4 + u][c] *= g;
                        d[u][c] = fmaf(kr[u], s[4 * i4 + u][c], d[u][c]);
                    }
                }
            }
            float dot[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) dot[c] = (d[0][c] + d[1][c]) + (d[2][c] + d[3][c]);
#pragma unroll
            for (int x = 1; x < kDeltaGroup; x <<= 1) {
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    dot[c] += __shfl_xor_sync(0xffffffffu, dot[c], x);
                    o_part[c] += __shfl_xor_sync(0xffffffffu, o_part[c], x);
                }
            }
            if (c0 + tt > 0) emit(s0 + c0 + tt - 1, o_part);
            float u_[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) u_[c] = beta * (s_v[stage][tt][my + c] - dot[c]);
            float e[4][CPT];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
#pragma unroll
                for (int c = 0; c < CPT; ++c) e[u][c] = 0.f;
            }
#pragma unroll
            for (int i4 = 0; i4 < RPT / 4; ++i4) {
                const float4 kk = k4[i4 * kDeltaGroup], qq = q4[i4 * kDeltaGroup];
                const float kr[4] = {kk.x, kk.y, kk.z, kk.w}, qr[4] = {qq.x, qq.y, qq.z, qq.w};
#pragma unroll
                for (int u = 0; u < 4; ++u) {
#pragma unroll
                    for (int c = 0; c < CPT; ++c) {
                        s[4 * i4 + u][c] = fmaf(kr[u], u_[c], s[4 * i4 + u][c]);
                        e[u][c] = fmaf(qr[u], s[4 * i4 + u][c], e[u][c]);
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < CPT; ++c) o_part[c] = (e[0][c] + e[1][c]) + (e[2][c] + e[3][c]);
        }
    }
    if (n > 0) {
#pragma unroll
        for (int x = 1; x < kDeltaGroup; x <<= 1) {
#pragma unroll
            for (int c = 0; c < CPT; ++c) o_part[c] += __shfl_xor_sync(0xffffffffu, o_part[c], x);
        }
        emit(s0 + n - 1, o_part);
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int row = (i / 4 * kDeltaGroup + rg) * 4 + i % 4;
        float* dst = S + static_cast<size_t>(row) * p.dv + col0 + my;
        if (CPT == 4 && vec) {
            if (row < p.dk && my < n_cols)
                *reinterpret_cast<float4*>(dst) = make_float4(s[i][0], s[i][CPT > 1 ? 1 : 0], s[i][CPT > 2 ? 2 : 0], s[i][CPT > 3 ? 3 : 0]);
        } else {
#pragma unroll
            for (int c = 0; c < CPT; ++c)
                if (row < p.dk && my + c < n_cols) dst[c] = s[i][c];
        }
    }
    // the convolution's last taps - 1 inputs of this request, a run of channels per block
    const int keep = p.taps - 1;
    if (keep > 0) {
        float* st = slot + p.conv_off;
        const int blocks = gridDim.x * gridDim.y, b = blockIdx.y * gridDim.x + blockIdx.x;
        const int run = (p.C + blocks - 1) / blocks;
        for (int c = b * run + tid; c < min(p.C, (b + 1) * run); c += kDeltaWarps * 32) {
            float vals[16];
            for (int j = 0; j < keep; ++j) {
                const int rel = n - keep + j;                 // index among the segment's rows; negative: an older input
                vals[j] = rel >= 0 ? p.proj[static_cast<size_t>(s0 + rel) * p.ld + p.in_off + c] : st[static_cast<size_t>(keep + rel) * p.C + c];
            }
            for (int j = 0; j < keep; ++j) st[static_cast<size_t>(j) * p.C + c] = vals[j];
        }
    }
}

template <int RPT>
static void launch_delta_scan(const DeltaArgs& a, int R, bool narrow, int wide, cudaStream_t st) {
    if (narrow) {
        constexpr unsigned cols = kDeltaWarps * (32 / kDeltaGroup);
        launch_kernel((delta_scan_kernel<RPT, 1>), dim3((a.dv + cols - 1) / cols, a.H, R), dim3(kDeltaWarps * 32), 0, st, a, wide);
    } else {
        constexpr unsigned cols = kDeltaWarps * (32 / kDeltaGroup) * 4;
        launch_kernel((delta_scan_kernel<RPT, 4>), dim3((a.dv + cols - 1) / cols, a.H, R), dim3(kDeltaWarps * 32), 0, st, a, wide);
    }
}

}  // namespace gi

using namespace gi;

// The whole mixer between its input and output products' neighbours: delta_prepare, then delta_scan. narrow: 1 spreads a
// head's columns over many warps (long portions), 0 keeps four columns a thread (steps of few tokens per request); the
// results are the same.
static int gi_gated_delta_impl(const float* proj, int ld, int in_off, int b_off, int a_off, const float* conv, int taps,
                               const float* a_log, const float* dt_bias, float q_scale, float unit_eps, float* state,
                               long long slot_stride, long long state_off, long long conv_off, const int* row_req,
                               const int* seg_start, const int* seg_len, const int* state_slots, float* qkv, float* gates,
                               float* out, int T, int R, int H, int G, int dk, int dv, int narrow, void* stream) {
    if (T == 0 || R == 0) return 0;
    GI_REQUIRE(T > 0 && R > 0 && H > 0 && G > 0 && dk > 0 && dv > 0, "gated_delta: sizes must be positive");
    GI_REQUIRE(H % G == 0, "gated_delta: %d heads are not a multiple of %d key heads", H, G);
    GI_REQUIRE(dk <= kDeltaMaxDim, "gated_delta: %d state rows per head exceed %d", dk, kDeltaMaxDim);
    GI_REQUIRE(taps >= 1 && taps <= 17, "gated_delta: %d convolution taps are not supported (1 to 17)", taps);
    const int C = 2 * G * dk + H * dv;
    GI_REQUIRE(in_off >= 0 && in_off + C <= ld && b_off >= 0 && b_off + H <= ld && a_off >= 0 && a_off + H <= ld,
               "gated_delta: the columns lie outside the input row of %d", ld);
    GI_REQUIRE(H <= 65535 && R <= 65535 && (T + kPrepTokens - 1) / kPrepTokens <= 65535, "gated_delta: the grid limit 65535 is exceeded");
    DeltaArgs a{proj, ld, in_off, b_off, a_off, conv, a_log, dt_bias, state, slot_stride, state_off, conv_off, row_req, seg_start,
                seg_len, state_slots, qkv, gates, out, T, H, G, dk, dv, C, taps, q_scale, unit_eps};
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const int items = 2 * G + (H * dv + 127) / 128 + 1;
    launch_kernel(delta_prepare_kernel, dim3((items + 7) / 8, (T + kPrepTokens - 1) / kPrepTokens), dim3(256), 0, st, a);
    if (check_launch("gated_delta (prepare)")) return 1;
    const int wide = dk % 4 == 0 && dv % 4 == 0 && reinterpret_cast<uintptr_t>(qkv) % 16 == 0;
    if (dk <= 32) launch_delta_scan<4>(a, R, narrow != 0, wide, st);
    else if (dk <= 64) launch_delta_scan<8>(a, R, narrow != 0, wide, st);
    else if (dk <= 96) launch_delta_scan<12>(a, R, narrow != 0, wide, st);
    else if (dk <= 128) launch_delta_scan<16>(a, R, narrow != 0, wide, st);
    else if (dk <= 192) launch_delta_scan<24>(a, R, narrow != 0, wide, st);
    else launch_delta_scan<32>(a, R, narrow != 0, wide, st);
    return check_launch("gated_delta");
}

extern "C" int gi_gated_delta(const float* proj, int ld, int in_off, int b_off, int a_off, const float* conv, int taps, const float* a_log, const float* dt_bias, float q_scale, float unit_eps, float* state, long long slot_stride, long long state_off, long long conv_off, const int* row_req, const int* seg_start, const int* seg_len, const int* state_slots, float* qkv, float* gates, float* out, int T, int R, int H, int G, int dk, int dv, int narrow, void* stream) {
    return gi::dispatch(gi_gated_delta_impl, proj, ld, in_off, b_off, a_off, conv, taps, a_log, dt_bias, q_scale, unit_eps, state, slot_stride, state_off, conv_off, row_req, seg_start, seg_len, state_slots, qkv, gates, out, T, R, H, G, dk, dv, narrow, stream);
}
