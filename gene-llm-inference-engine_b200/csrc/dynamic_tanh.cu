// The norm that computes no mean or variance, N(x) = tanh(alpha x) * w + b with one number alpha per norm, and the pass
// over the residual stream of a layer that has such a norm before and after each sublayer.
//
//   dynamic_tanh      out[r] = N(x[row_r]) for all rows or for listed ones
//   add_dynamic_tanh  x += N(y) (+ more) and y = 0, and in the same pass what runs next reads: N'(x) in the compute dtype.
//                     y: what a sublayer added its output to; ``more``: rows added to the stream ahead of what runs next
//
// All arithmetic is 32-bit; only stores round. A value depends on its own place only, so rows are cut as it suits memory:
// four values to a thread with 16-byte accesses where the width allows it.
#include "common.cuh"

namespace gi {

struct TanhNorm {
    float alpha;
    const float* w; const float* b;
};

template <int VEC> struct Values { float v[VEC]; };
template <int VEC>
__device__ __forceinline__ Values<VEC> load_values(const float* p) {
    Values<VEC> r;
    if constexpr (VEC == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        r.v[0] = q.x; r.v[1] = q.y; r.v[2] = q.z; r.v[3] = q.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VEC>
__device__ __forceinline__ void store_values(float* p, const Values<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VEC>
__device__ __forceinline__ void store_values(__nv_bfloat16* p, const Values<VEC>& r) {
    if constexpr (VEC == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<const uint32_t*>(&lo);
        raw.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = raw;
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}
template <int VEC>
__device__ __forceinline__ Values<VEC> norm_of(const TanhNorm& n, const Values<VEC>& x, int c) {
    const Values<VEC> w = load_values<VEC>(n.w + c), b = load_values<VEC>(n.b + c);
    Values<VEC> r;
#pragma unroll
    for (int e = 0; e < VEC; ++e) r.v[e] = fmaf(tanhf(n.alpha * x.v[e]), w.v[e], b.v[e]);
    return r;
}

template <int VEC, typename TOut>
__global__ void __launch_bounds__(256)
dynamic_tanh_kernel(const float* __restrict__ x, const int* __restrict__ rows, const TanhNorm n, TOut* __restrict__ out, int D, size_t total) {
    pdl_prologue();
    const size_t i = (static_cast<size_t>(blockIdx.x) * 256 + threadIdx.x) * VEC;
    if (i >= total) return;
    const size_t r = i / D;
    const int c = static_cast<int>(i % D);
    const size_t src = rows ? static_cast<size_t>(rows[r]) : r;
    store_values<VEC>(out + i, norm_of<VEC>(n, load_values<VEC>(x + src * D + c), c));
}

template <int VEC, typename TOut>
__global__ void __launch_bounds__(256)
add_dynamic_tanh_kernel(float* __restrict__ y, const TanhNorm n, float* __restrict__ x, const float* __restrict__ more,
                        const TanhNorm next, TOut* __restrict__ xn, int D, size_t total, int clear) {
    pdl_prologue();
    const size_t i = (static_cast<size_t>(blockIdx.x) * 256 + threadIdx.x) * VEC;
    if (i >= total) return;
    const int c = static_cast<int>(i % D);
    Values<VEC> v = load_values<VEC>(x + i), z;
    Values<VEC> a = load_values<VEC>(y + i);
    if (more) z = load_values<VEC>(more + i);
    a = norm_of<VEC>(n, a, c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        v.v[e] += a.v[e];
        if (more) v.v[e] += z.v[e];
    }
    store_values<VEC>(x + i, v);
    if (clear) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) a.v[e] = 0.f;
        store_values<VEC>(y + i, a);
    }
    if (xn) store_values<VEC>(xn + i, norm_of<VEC>(next, v, c));
}

static bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

}  // namespace gi

using namespace gi;

static int gi_dynamic_tanh_impl(const float* x, const int* rows, float alpha, const float* w, const float* b, void* out, int out_dtype,
                                int n_rows, int D, void* stream) {
    if (n_rows == 0) return 0;
    GI_REQUIRE(n_rows > 0 && D > 0, "dynamic_tanh: sizes must be positive (rows=%d, D=%d)", n_rows, D);
    GI_REQUIRE(out_dtype == kF32 || out_dtype == kBF16, "dynamic_tanh: unsupported output dtype code %d", out_dtype);
    const size_t total = static_cast<size_t>(n_rows) * D;
    const bool vec = D % 4 == 0 && aligned16(x) && aligned16(w) && aligned16(b) && aligned16(out);
    const size_t blocks = (total / (vec ? 4 : 1) + 255) / 256;
    GI_REQUIRE(blocks <= 2147483647u, "dynamic_tanh: too many rows");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const TanhNorm n{alpha, w, b};
    const dim3 grid(static_cast<unsigned>(blocks));
    if (out_dtype == kBF16) {
        auto* o = static_cast<__nv_bfloat16*>(out);
        if (vec) launch_kernel((dynamic_tanh_kernel<4, __nv_bfloat16>), grid, dim3(256), 0, st, x, rows, n, o, D, total);
        else launch_kernel((dynamic_tanh_kernel<1, __nv_bfloat16>), grid, dim3(256), 0, st, x, rows, n, o, D, total);
    } else {
        auto* o = static_cast<float*>(out);
        if (vec) launch_kernel((dynamic_tanh_kernel<4, float>), grid, dim3(256), 0, st, x, rows, n, o, D, total);
        else launch_kernel((dynamic_tanh_kernel<1, float>), grid, dim3(256), 0, st, x, rows, n, o, D, total);
    }
    return check_launch("dynamic_tanh");
}

static int gi_add_dynamic_tanh_impl(float* y, float alpha, const float* w, const float* b, float* x, const float* more, float next_alpha,
                                    const float* next_w, const float* next_b, void* xn, int xn_dtype, int n_rows, int D, int clear,
                                    void* stream) {
    if (n_rows == 0) return 0;
    GI_REQUIRE(n_rows > 0 && D > 0, "add_dynamic_tanh: sizes must be positive (rows=%d, D=%d)", n_rows, D);
    GI_REQUIRE(xn == nullptr || (next_w && next_b), "add_dynamic_tanh: the next norm's weight and bias are missing");
    GI_REQUIRE(xn_dtype == kF32 || xn_dtype == kBF16, "add_dynamic_tanh: unsupported dtype code %d", xn_dtype);
    const size_t total = static_cast<size_t>(n_rows) * D;
    const bool vec = D % 4 == 0 && aligned16(y) && aligned16(w) && aligned16(b) && aligned16(x) && aligned16(more) && aligned16(next_w) &&
                     aligned16(next_b) && aligned16(xn);
    const size_t blocks = (total / (vec ? 4 : 1) + 255) / 256;
    GI_REQUIRE(blocks <= 2147483647u, "add_dynamic_tanh: too many rows");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const TanhNorm n{alpha, w, b}, next{next_alpha, next_w, next_b};
    const dim3 grid(static_cast<unsigned>(blocks));
    if (xn_dtype == kBF16) {
        auto* o = static_cast<__nv_bfloat16*>(xn);
        if (vec) launch_kernel((add_dynamic_tanh_kernel<4, __nv_bfloat16>), grid, dim3(256), 0, st, y, n, x, more, next, o, D, total, clear);
        else launch_kernel((add_dynamic_tanh_kernel<1, __nv_bfloat16>), grid, dim3(256), 0, st, y, n, x, more, next, o, D, total, clear);
    } else {
        auto* o = static_cast<float*>(xn);
        if (vec) launch_kernel((add_dynamic_tanh_kernel<4, float>), grid, dim3(256), 0, st, y, n, x, more, next, o, D, total, clear);
        else launch_kernel((add_dynamic_tanh_kernel<1, float>), grid, dim3(256), 0, st, y, n, x, more, next, o, D, total, clear);
    }
    return check_launch("add_dynamic_tanh");
}

extern "C" int gi_dynamic_tanh(const float* x, const int* rows, float alpha, const float* w, const float* b, void* out, int out_dtype,
                               int n_rows, int D, void* stream) {
    return gi::dispatch(gi_dynamic_tanh_impl, x, rows, alpha, w, b, out, out_dtype, n_rows, D, stream);
}

extern "C" int gi_add_dynamic_tanh(float* y, float alpha, const float* w, const float* b, float* x, const float* more, float next_alpha,
                                   const float* next_w, const float* next_b, void* xn, int xn_dtype, int n_rows, int D, int clear,
                                   void* stream) {
    return gi::dispatch(gi_add_dynamic_tanh_impl, y, alpha, w, b, x, more, next_alpha, next_w, next_b, xn, xn_dtype, n_rows, D, clear, stream);
}
