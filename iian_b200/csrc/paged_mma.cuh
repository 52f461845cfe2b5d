// Shared by the attention kernels that walk a paged K/V cache with mma.sync: asynchronous copies, fragment loads, the products,
// shared-memory layouts of a tile of 64 keys, bounded mbarrier waits, TMA copies of pages and their tensor maps.
#pragma once
#include <cuda.h>

#include "common.cuh"
#include <mutex>

namespace iian {

constexpr int BN = 64;   // keys per tile

// Tensor maps of the K and V caches for the TMA form of the decode kernel (unused by the other forms).
struct KvMaps {
    CUtensorMap k, v;
};

__device__ __forceinline__ unsigned smem_u32(const void * p) { return (unsigned) __cvta_generic_to_shared(p); }

__device__ __forceinline__ void cp_async16(unsigned dst, const void * src, bool valid) {
    const int n = valid ? 16 : 0;   // src-size 0: the 16 bytes are zero-filled, nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N)); }

__device__ __forceinline__ void ldmatrix_x4(unsigned & r0, unsigned & r1, unsigned & r2, unsigned & r3, unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned & r0, unsigned & r1, unsigned & r2, unsigned & r3, unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float * c, const unsigned * a, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 2^x in one MUFU instruction (about 2 ulp; -inf gives 0).  The probabilities are rounded to bfloat16 next.
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// tanh(x) as 1 - 2 / (1 + e^2x) from the hardware's exponential and reciprocal, absolute error of a few 1e-7
__device__ __forceinline__ float score_tanh(float x) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * 2.8853900817779268f));        // e^2x
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
    return fmaf(-2.0f, r, 1.0f);
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<unsigned *>(&v);
}

// byte offset of 16-byte chunk `chunk` of row `row` in a tile with rows of HD bf16, XOR-swizzled so that
// the 8 rows an ldmatrix touches fall into different banks
template <int HD> __device__ __forceinline__ unsigned swz(int row, int chunk) {
    return (unsigned) (row * HD * 2 + ((chunk ^ (row & 7)) << 4));
}

// The same for a tile that TMA wrote with its 128-byte swizzle (head size 128): two planes of 128-byte rows,
// one per half of the head, chunks XOR-swizzled within a row by the row's low three bits.
template <int HD, bool TMA> __device__ __forceinline__ unsigned kv_off(int row, int chunk) {
    if (TMA) return (unsigned) ((chunk >> 3) * (BN * 128) + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
    return swz<HD>(row, chunk);
}

constexpr unsigned kDecodeSpinLimit = 4u * 1000u * 1000u;
__device__ __forceinline__ void dk_mbar_init(unsigned bar, unsigned count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count));
}
__device__ __forceinline__ void dk_expect_tx(unsigned bar, unsigned bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ bool dk_wait(unsigned bar, unsigned parity) {          // bounded: false when it gave up
    for (unsigned spin = 0; spin < kDecodeSpinLimit; spin++) {
        unsigned done;
        asm volatile("{\n .reg .pred p;\n mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}"
                     : "=r"(done) : "r"(bar), "r"(parity) : "memory");
        if (done) return true;
    }
    return false;
}
__device__ __forceinline__ void dk_tma_4d(unsigned dst, const CUtensorMap * map, int x, int y, int z, int w, unsigned bar) {
    asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];"
                 ::"r"(dst), "l"(map), "r"(x), "r"(y), "r"(z), "r"(w), "r"(bar) : "memory");
}

typedef CUresult (*KvEncodeFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                               const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// Tensor map of a cache [num_pages, nkv, page_size, 128] bf16 with boxes of one page and half a head
// ([page_size rows, 64 values], 128-byte swizzle).  The maps of the caches seen so far are kept (a cache keeps its
// address for the life of an engine), so that a launch costs no call into the driver.
static int kv_map_for(const void * base, int num_pages, int nkv, int page_size, CUtensorMap * out) {
    struct Entry { const void * base; int num_pages, nkv, page_size; CUtensorMap map; };
    static Entry cache[256];
    static int n_cached = 0, next = 0;
    static std::mutex mu;
    std::lock_guard<std::mutex> lock(mu);
    for (int i = 0; i < n_cached; i++) {
        const Entry & e = cache[i];
        if (e.base == base && e.num_pages == num_pages && e.nkv == nkv && e.page_size == page_size) { *out = e.map; return IIAN_OK; }
    }
    static KvEncodeFn fn = nullptr;
    if (fn == nullptr) {
        void * f = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &f, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
            return IIAN_ERR_LIMIT;
        fn = (KvEncodeFn) f;
    }
    cuuint64_t dims[4] = {128, (cuuint64_t) page_size, (cuuint64_t) nkv, (cuuint64_t) num_pages};
    cuuint64_t strides[3] = {256, (cuuint64_t) page_size * 256, (cuuint64_t) nkv * page_size * 256};
    cuuint32_t box[4] = {64, (cuuint32_t) page_size, 1, 1};
    cuuint32_t estr[4] = {1, 1, 1, 1};
    CUtensorMap map;
    CUresult r = fn(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void *>(base), dims, strides, box, estr,
                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                    CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) return 2000 + (int) r;
    Entry & e = cache[next];
    e.base = base; e.num_pages = num_pages; e.nkv = nkv; e.page_size = page_size; e.map = map;
    next = (next + 1) % 256;
    if (n_cached < 256) n_cached++;
    *out = map;
    return IIAN_OK;
}

static int decode_sm_count() {
    static int n[64] = {};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 148;
    if (n[dev] == 0) {
        int v = 0;
        if (cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || v <= 0) v = 148;
        n[dev] = v;
    }
    return n[dev];
}

}  // namespace iian
