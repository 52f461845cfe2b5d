// Row-wise kernels of a norm that takes no statistics of its row: n(x) = w tanh(alpha x) + b, one alpha per norm.
//
//   tanh_add_tanh   x += u tanh(alpha_y y) + c [+ r]   (a sub-layer output that passes such a norm on its way into the float32
//                   stream; without u it is added as it is; r: one float32 vector that every row gets),
//                   then out = w tanh(alpha x) + b   (each of y, r, out optional)
//   add_row         x += r for every row
//
// `A` is the activation type; the stream, the norms and the sums are float32.  Every element depends on its own column only.
#include "common.cuh"

namespace iian {

constexpr int kTanhThreads = 256;

__device__ __forceinline__ float4 tn_load4(const float * p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 tn_load4(const __nv_bfloat16 * p) {
    const uint2 raw = *reinterpret_cast<const uint2 *>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void tn_store4(float * p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void tn_store4(__nv_bfloat16 * p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<unsigned *>(&a);
    raw.y = *reinterpret_cast<unsigned *>(&b);
    *reinterpret_cast<uint2 *>(p) = raw;
}

struct TanhNormArgs {
    float * residual;           // [N, H]
    const void * y;             // [N, H] or null
    float alpha_y;
    const float * u, * c;       // [H] or null (then y is added as it is)
    const float * row;          // [H] or null
    float alpha;
    const float * w, * b;       // [H]
    void * out;                 // [N, H] or null
    long long total;
    int H;
};

// one column of a row: x is the stream's entry (updated), the result what the next product reads
__device__ __forceinline__ float tn_one(float & x, bool has_y, float y, float alpha_y, bool normed, float u, float c, float r,
                                        bool want, float alpha, float w, float b) {
    if (has_y) x += normed ? fmaf(u, tanhf(alpha_y * y), c) : y;
    x += r;
    return want ? fmaf(w, tanhf(alpha * x), b) : 0.0f;
}

template <typename A>
__global__ void __launch_bounds__(kTanhThreads) tanh_add_tanh_kernel(const TanhNormArgs p) {
    pdl_wait();
    pdl_launch_dependents();
    const long long e = (long long) blockIdx.x * kTanhThreads + threadIdx.x;
    if (e >= p.total) return;
    const int i = (int) (e % p.H);
    const A * yp = (const A *) p.y;
    float x = p.residual[e];
    const bool normed = p.u != nullptr;
    const float o = tn_one(x, yp != nullptr, yp != nullptr ? to_f32(yp[e]) : 0.0f, p.alpha_y, normed, normed ? p.u[i] : 0.0f,
                           normed ? p.c[i] : 0.0f, p.row != nullptr ? p.row[i] : 0.0f, p.out != nullptr, p.alpha,
                           p.out != nullptr ? p.w[i] : 0.0f, p.out != nullptr ? p.b[i] : 0.0f);
    if (yp != nullptr || p.row != nullptr) p.residual[e] = x;
    if (p.out != nullptr) ((A *) p.out)[e] = from_f32<A>(o);
}

// The same four columns at a time (H a multiple of 4, every pointer aligned to four entries).  Grid (column blocks, row
// groups): a thread keeps its columns' weights in registers and walks the rows of its group.
template <typename A, bool HAS_Y, bool HAS_OUT>
__global__ void __launch_bounds__(kTanhThreads) tanh_add_tanh_vec_kernel(const TanhNormArgs p, int N, int rows_per_block) {
    pdl_wait();
    pdl_launch_dependents();
    const int i = 4 * (blockIdx.x * blockDim.x + threadIdx.x);
    if (i >= p.H) return;
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    const bool normed = p.u != nullptr;
    const float4 u = normed ? tn_load4(p.u + i) : zero, c = normed ? tn_load4(p.c + i) : zero;
    const float4 r = p.row != nullptr ? tn_load4(p.row + i) : zero;
    const float4 w = HAS_OUT ? tn_load4(p.w + i) : zero, b = HAS_OUT ? tn_load4(p.b + i) : zero;
    const int t0 = blockIdx.y * rows_per_block, t1 = min(N, t0 + rows_per_block);
    for (int t = t0; t < t1; t++) {
        const size_t e = (size_t) t * p.H + i;
        float4 x = tn_load4(p.residual + e), y = zero;
        if (HAS_Y) y = tn_load4((const A *) p.y + e);
        float4 o;
        o.x = tn_one(x.x, HAS_Y, y.x, p.alpha_y, normed, u.x, c.x, r.x, HAS_OUT, p.alpha, w.x, b.x);
        o.y = tn_one(x.y, HAS_Y, y.y, p.alpha_y, normed, u.y, c.y, r.y, HAS_OUT, p.alpha, w.y, b.y);
        o.z = tn_one(x.z, HAS_Y, y.z, p.alpha_y, normed, u.z, c.z, r.z, HAS_OUT, p.alpha, w.z, b.z);
        o.w = tn_one(x.w, HAS_Y, y.w, p.alpha_y, normed, u.w, c.w, r.w, HAS_OUT, p.alpha, w.w, b.w);
        if (HAS_Y || p.row != nullptr) tn_store4(p.residual + e, x);
        if (HAS_OUT) tn_store4((A *) p.out + e, o);
    }
}

template <typename A>
static int launch_tanh(const TanhNormArgs & a, int N, cudaStream_t stream) {
    const uintptr_t act = 4 * sizeof(A);
    const bool vec = a.H % 4 == 0 && ((uintptr_t) a.residual | (uintptr_t) a.u | (uintptr_t) a.c | (uintptr_t) a.row | (uintptr_t) a.w |
                                      (uintptr_t) a.b) % 16 == 0 && ((uintptr_t) a.y | (uintptr_t) a.out) % act == 0;
    if (!vec) {
        const unsigned blocks = (unsigned) ((a.total + kTanhThreads - 1) / kTanhThreads);
        return iian_launch(tanh_add_tanh_kernel<A>, dim3(blocks), dim3(kTanhThreads), 0, stream, a);
    }
    const int quads = a.H / 4;
    const int threads = quads >= kTanhThreads ? kTanhThreads : (quads + 31) / 32 * 32;
    const int bx = (quads + threads - 1) / threads;
    // few rows: one each, so that they spread over the GPU; many: a few per block, so that weights are read once for them
    int per = (int) (((long long) N * bx) / 2368);             // 148 SMs x 16 blocks
    per = per < 1 ? 1 : per > 8 ? 8 : per;
    while ((N + per - 1) / per > 65535) per *= 2;
    const dim3 grid(bx, (N + per - 1) / per);
    if (a.y != nullptr && a.out != nullptr) return iian_launch(tanh_add_tanh_vec_kernel<A, true, true>, grid, dim3(threads), 0, stream, a, N, per);
    if (a.y != nullptr) return iian_launch(tanh_add_tanh_vec_kernel<A, true, false>, grid, dim3(threads), 0, stream, a, N, per);
    if (a.out != nullptr) return iian_launch(tanh_add_tanh_vec_kernel<A, false, true>, grid, dim3(threads), 0, stream, a, N, per);
    return iian_launch(tanh_add_tanh_vec_kernel<A, false, false>, grid, dim3(threads), 0, stream, a, N, per);
}

}  // namespace iian

using namespace iian;

// residual: f32 [N, H] in place; y: A [N, H] or null; u, c: f32 [H], both or neither; row: f32 [H] or null; w, b: f32 [H] and
// out: A [N, H], all or none.  add_row is this with `row` alone.
IIAN_API int iian_tanh_add_tanh(float * residual, const void * y, float alpha_y, const float * u, const float * c, const float * row,
                                float alpha, const float * w, const float * b, void * out, int act_dtype, int N, int H,
                                cudaStream_t stream) {
    if (N <= 0) return IIAN_OK;
    if (H <= 0 || (u == nullptr) != (c == nullptr) || (out != nullptr && (w == nullptr || b == nullptr))) return IIAN_ERR_SHAPE;
    if (y == nullptr && u != nullptr) return IIAN_ERR_SHAPE;
    if (y == nullptr && row == nullptr && out == nullptr) return IIAN_OK;
    TanhNormArgs a;
    a.residual = residual; a.y = y; a.alpha_y = alpha_y; a.u = u; a.c = c; a.row = row; a.alpha = alpha; a.w = out != nullptr ? w : nullptr;
    a.b = out != nullptr ? b : nullptr; a.out = out; a.total = (long long) N * H; a.H = H;
    if (act_dtype == IIAN_F32) return launch_tanh<float>(a, N, stream);
    if (act_dtype == IIAN_BF16) return launch_tanh<__nv_bfloat16>(a, N, stream);
    return IIAN_ERR_DTYPE;
}
