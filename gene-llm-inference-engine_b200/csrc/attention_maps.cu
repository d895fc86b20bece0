// Attention whose heads have two score maps over the same values, the second taken off the first.
//
//   maps_norm_store   from the 32-bit projections of a token: every query and key head is [map 1, map 2] of dim values each;
//                     each map is brought to unit RMS and weighted, queries are multiplied by a factor that grows with the
//                     position, 1 + coef ln(floor((p + 1) / every) + 1). Keys go to the token's page row as they are,
//                     [map 1, map 2] in one row, values beside them. A query head becomes two rows, [map 1, 0] and
//                     [0, map 2]: the scores of row m against the key rows are then those of map m, and any attention kernel
//                     over (2 H query heads, G key heads) computes both maps, which share every key and value row they
//                     read. Rows may be wider than 2 dim (values: than their own width), with zeros behind, so that the
//                     attention kernels that are built for a few widths serve other sizes too
//   maps_combine      o = a1 - lambda a2 per head, brought to unit RMS over the value width, times a constant
//
// All arithmetic is 32-bit; only stores round. A row's result depends on that row only.
#include "common.cuh"

namespace gi {

constexpr int kMapsWarps = 4;
constexpr int kMapsMaxDim = 512;

// A warp per (head, map): query heads first, then key heads (whose first map also carries the head's values).
template <typename T>
__global__ void __launch_bounds__(kMapsWarps * 32)
maps_norm_store_kernel(const float* __restrict__ in, int ld, int q_off, int k_off, int v_off, const float* __restrict__ q_norm,
                       const float* __restrict__ k_norm, float eps, float temp_coef, float temp_every,
                       const int* __restrict__ positions, const int* __restrict__ row_req, const int* __restrict__ block_tables,
                       int table_stride, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache, int H, int G,
                       int dim, int vd, int row_width, int v_row, int page_size, int write_kv) {
    pdl_prologue();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int pos = positions[t];
    const float* row = in + static_cast<size_t>(t) * ld;
    const float temp = temp_coef != 0.f ? 1.0f + temp_coef * logf(floorf(static_cast<float>(pos + 1) / temp_every) + 1.0f) : 1.0f;
    size_t page_row = 0;
    if (write_kv) {
        const int page = block_tables[static_cast<size_t>(row_req[t]) * table_stride + pos / page_size];
        page_row = static_cast<size_t>(page) * G * page_size + pos % page_size;
    }
    const int n_items = 2 * (H + (write_kv ? G : 0));
    for (int item = blockIdx.y * kMapsWarps + warp; item < n_items; item += kMapsWarps * gridDim.y) {
        const int head = item >> 1, map = item & 1;
        const bool is_q = head < H;
        const float* src = row + (is_q ? q_off + item * dim : k_off + (item - 2 * H) * dim);
        const float* w = is_q ? q_norm : k_norm;
        float ss = 0.f;
        for (int i = lane; i < dim; i += 32) ss = fmaf(src[i], src[i], ss);
        ss = warp_sum(ss);
        const float scale = 1.0f / sqrtf(ss / static_cast<float>(dim) + eps);
        if (is_q) {
            T* dst = q_out + (static_cast<size_t>(t) * 2 * H + item) * row_width;
            for (int d = lane; d < row_width; d += 32) {
                const int i = d - map * dim;
                dst[d] = from_float<T>(i >= 0 && i < dim ? w[i] * (scale * src[i]) * temp : 0.f);
            }
        } else {
            const size_t at = page_row + static_cast<size_t>(head - H) * page_size;
            T* dst = k_cache + at * row_width + map * dim;
            const int n = map == 0 ? dim : row_width - dim;                  // the second map writes the zeros behind it, too
            for (int i = lane; i < n; i += 32) dst[i] = from_float<T>(i < dim ? w[i] * (scale * src[i]) : 0.f);
            if (map == 0) {
                const float* vsrc = row + v_off + (head - H) * vd;
                T* vdst = v_cache + at * v_row;
                for (int d = lane; d < v_row; d += 32) vdst[d] = from_float<T>(d < vd ? vsrc[d] : 0.f);
            }
        }
    }
}

// A warp per (token, head); up to 512 value dimensions stay in registers between the sum and the scaling.
template <typename TIn, typename TOut>
__global__ void __launch_bounds__(256)
maps_combine_kernel(const TIn* __restrict__ a, TOut* __restrict__ out, float lambda, float eps, float factor, int vd, int v_row,
                    long long heads) {
    pdl_prologue();
    const long long item = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
    if (item >= heads) return;
    const int lane = threadIdx.x & 31;
    const TIn* a1 = a + item * 2 * v_row;
    const TIn* a2 = a1 + v_row;
    float o[kMapsMaxDim / 32];
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < kMapsMaxDim / 32; ++u) {
        const int d = lane + 32 * u;
        o[u] = d < vd ? to_float(a1[d]) - lambda * to_float(a2[d]) : 0.f;
        ss = fmaf(o[u], o[u], ss);
    }
    ss = warp_sum(ss);
    const float f = factor / sqrtf(ss / static_cast<float>(vd) + eps);
#pragma unroll
    for (int u = 0; u < kMapsMaxDim / 32; ++u)
        if (lane + 32 * u < vd) out[item * vd + lane + 32 * u] = from_float<TOut>(o[u] * f);
}

}  // namespace gi

using namespace gi;

static int gi_maps_norm_store_impl(const float* in, int ld, int q_off, int k_off, int v_off, const float* q_norm, const float* k_norm,
                                   float eps, float temp_coef, float temp_every, const int* positions, const int* row_req,
                                   const int* block_tables, int table_stride, void* q_out, void* k_cache, void* v_cache, int dtype,
                                   int T, int H, int G, int dim, int vd, int row_width, int v_row, int page_size, int write_kv, void* stream) {
    if (T == 0) return 0;
    GI_REQUIRE(T > 0 && H > 0 && G > 0 && dim > 0 && vd > 0 && page_size > 0, "maps_norm_store: sizes must be positive");
    GI_REQUIRE(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + 2 * H * dim <= ld && k_off + 2 * G * dim <= ld && v_off + G * vd <= ld,
               "maps_norm_store: the columns of queries, keys or values lie outside the input row of %d", ld);
    GI_REQUIRE(row_width >= 2 * dim && v_row >= vd, "maps_norm_store: a row is shorter than what it holds");
    GI_REQUIRE(temp_coef == 0.f || temp_every > 0.f, "maps_norm_store: the blocks of the query factor must have a positive length");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const int items = 2 * (H + G);
    // few rows (decoding): the heads of a token are spread over blocks; many rows: a few blocks per token
    const unsigned by = static_cast<unsigned>(std::min((items + kMapsWarps - 1) / kMapsWarps, T >= 256 ? 2 : 65535));
    if (dtype == kF32)
        launch_kernel((maps_norm_store_kernel<float>), dim3(T, by), dim3(kMapsWarps * 32), 0, st, in, ld, q_off, k_off, v_off, q_norm, k_norm, eps,
                      temp_coef, temp_every, positions, row_req, block_tables, table_stride, static_cast<float*>(q_out),
                      static_cast<float*>(k_cache), static_cast<float*>(v_cache), H, G, dim, vd, row_width, v_row, page_size, write_kv);
    else if (dtype == kBF16)
        launch_kernel((maps_norm_store_kernel<__nv_bfloat16>), dim3(T, by), dim3(kMapsWarps * 32), 0, st, in, ld, q_off, k_off, v_off, q_norm, k_norm,
                      eps, temp_coef, temp_every, positions, row_req, block_tables, table_stride, static_cast<__nv_bfloat16*>(q_out),
                      static_cast<__nv_bfloat16*>(k_cache), static_cast<__nv_bfloat16*>(v_cache), H, G, dim, vd, row_width, v_row, page_size, write_kv);
    else
        GI_REQUIRE(false, "maps_norm_store: unsupported dtype code %d", dtype);
    return check_launch("maps_norm_store");
}

static int gi_maps_combine_impl(const void* a, int a_dtype, void* out, int out_dtype, float lambda, float eps, float factor, int T, int H,
                                int vd, int v_row, void* stream) {
    if (T == 0) return 0;
    GI_REQUIRE(T > 0 && H > 0 && vd > 0 && vd <= kMapsMaxDim, "maps_combine: a value size of %d is not supported (up to %d)", vd, kMapsMaxDim);
    GI_REQUIRE(v_row >= vd, "maps_combine: rows of %d hold no %d values", v_row, vd);
    GI_REQUIRE((a_dtype == kF32 || a_dtype == kBF16) && (out_dtype == kF32 || out_dtype == kBF16), "maps_combine: unsupported dtype code");
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const long long heads = static_cast<long long>(T) * H;
    const dim3 grid(static_cast<unsigned>((heads + 7) / 8));
    using bf = __nv_bfloat16;
    if (a_dtype == kF32 && out_dtype == kF32) launch_kernel((maps_combine_kernel<float, float>), grid, dim3(256), 0, st, static_cast<const float*>(a), static_cast<float*>(out), lambda, eps, factor, vd, v_row, heads);
    else if (a_dtype == kF32) launch_kernel((maps_combine_kernel<float, bf>), grid, dim3(256), 0, st, static_cast<const float*>(a), static_cast<bf*>(out), lambda, eps, factor, vd, v_row, heads);
    else if (out_dtype == kF32) launch_kernel((maps_combine_kernel<bf, float>), grid, dim3(256), 0, st, static_cast<const bf*>(a), static_cast<float*>(out), lambda, eps, factor, vd, v_row, heads);
    else launch_kernel((maps_combine_kernel<bf, bf>), grid, dim3(256), 0, st, static_cast<const bf*>(a), static_cast<bf*>(out), lambda, eps, factor, vd, v_row, heads);
    return check_launch("maps_combine");
}

extern "C" int gi_maps_norm_store(const float* in, int ld, int q_off, int k_off, int v_off, const float* q_norm, const float* k_norm, float eps, float temp_coef, float temp_every, const int* positions, const int* row_req, const int* block_tables, int table_stride, void* q_out, void* k_cache, void* v_cache, int dtype, int T, int H, int G, int dim, int vd, int row_width, int v_row, int page_size, int write_kv, void* stream) {
    return gi::dispatch(gi_maps_norm_store_impl, in, ld, q_off, k_off, v_off, q_norm, k_norm, eps, temp_coef, temp_every, positions, row_req, block_tables, table_stride, q_out, k_cache, v_cache, dtype, T, H, G, dim, vd, row_width, v_row, page_size, write_kv, stream);
}

extern "C" int gi_maps_combine(const void* a, int a_dtype, void* out, int out_dtype, float lambda, float eps, float factor, int T, int H, int vd, int v_row, void* stream) {
    return gi::dispatch(gi_maps_combine_impl, a, a_dtype, out, out_dtype, lambda, eps, factor, T, H, vd, v_row, stream);
}
