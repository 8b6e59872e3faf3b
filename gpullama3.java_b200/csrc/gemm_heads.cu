// One small product per head in one launch, bfloat16 on the tensor cores (mma.sync m16n8k16):
//     C[:, h n .. (h + 1) n) = A[:, h k .. (h + 1) k) W[h]^T          A [M, H k], W [H, n, k], C [M, H n]
// as latent attention needs on its way into and out of the latent space, where k and n are a head's sizes (a hundred or so) and the
// whole of K fits into shared memory.  A CTA takes 64 rows, one head and up to 128 of its columns: both tiles are fetched at once
// (cp.async, 16 bytes), four warps of 16 rows multiply, and the results leave through shared memory as whole 16-byte pieces where
// sizes and pointers allow.  Sums are 32-bit.  The work is a few bytes per flop: several CTAs per SM overlap their loads.
#include "run_tiles.cuh"

namespace b200 {

constexpr int kHeadCols = 128;

struct HeadProductArgs {
    const __nv_bfloat16* a;
    const __nv_bfloat16* w;
    __nv_bfloat16* c;
    int lda, ldc, M, n, k, wide_stores;
};

__global__ void __launch_bounds__(kRunThreads)
gemm_heads_kernel(HeadProductArgs p) {
    extern __shared__ __align__(16) uint8_t head_smem[];
    const int k_pad = (p.k + 15) / 16 * 16, ld = k_pad + 8;
    __nv_bfloat16* as = reinterpret_cast<__nv_bfloat16*>(head_smem);     // [kRun][ld]
    __nv_bfloat16* ws = as + kRun * ld;                                  // [kHeadCols][ld]
    const int h = blockIdx.z, m0 = blockIdx.x * kRun, n0 = blockIdx.y * kHeadCols;
    const int rows = min(kRun, p.M - m0), cols = min(kHeadCols, p.n - n0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3, mr = lane & 7, gq = lane >> 2, tq = lane & 3;
    const int per_row = k_pad / 8;
    pdl_launch_dependents();
    // (weights are written by no kernel: they are on their way before the dependency wait)
    const __nv_bfloat16* wh = p.w + ((size_t)h * p.n + n0) * p.k;
    for (int i = threadIdx.x; i < kHeadCols * per_row; i += kRunThreads) {
        const int r = i / per_row, c = (i % per_row) * 8;
        const bool take = r < cols && c < p.k;
        copy_16(ws + (size_t)r * ld + c, take ? wh + (size_t)r * p.k + c : p.w, take);
    }
    pdl_wait();
    const __nv_bfloat16* ah = p.a + (size_t)m0 * p.lda + (size_t)h * p.k;
    for (int i = threadIdx.x; i < kRun * per_row; i += kRunThreads) {
        const int r = i / per_row, c = (i % per_row) * 8;
        const bool take = r < rows && c < p.k;
        copy_16(as + (size_t)r * ld + c, take ? ah + (size_t)r * p.lda + c : p.a, take);
    }
    copies_done();
    __syncthreads();
    const int row0 = warp * 16;
    float acc[kHeadCols / 8][4];
#pragma unroll
    for (int j = 0; j < kHeadCols / 8; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
    if (row0 < rows) {
        for (int kk = 0; kk < k_pad / 16; ++kk) {
            uint32_t fa[4];
            ldsm4(fa, as + (row0 + (mi & 1) * 8 + mr) * ld + kk * 16 + (mi >> 1) * 8);
#pragma unroll
            for (int j = 0; j < kHeadCols / 16; ++j) {
                if (j * 16 >= cols) break;
                uint32_t fb[4];
                ldsm4(fb, ws + (j * 16 + (mi >> 1) * 8 + mr) * ld + kk * 16 + (mi & 1) * 8);
                mma_run(acc[2 * j], fa, fb[0], fb[1]);
                mma_run(acc[2 * j + 1], fa, fb[2], fb[3]);
            }
        }
    }
    __nv_bfloat16* out = p.c + (size_t)m0 * p.ldc + (size_t)h * p.n + n0;
    if (!p.wide_stores) {
        if (row0 >= rows) return;
#pragma unroll
        for (int j = 0; j < kHeadCols / 8; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = row0 + gq + (i >> 1) * 8, c = j * 8 + 2 * tq + (i & 1);
                if (r < rows && c < cols) out[(size_t)r * p.ldc + c] = __float2bfloat16_rn(acc[j][i]);
            }
        return;
    }
    __syncthreads();           // (the operands have been read: the results take their place)
    constexpr int ldo = kHeadCols + 8;
    __nv_bfloat16* os = reinterpret_cast<__nv_bfloat16*>(head_smem);
    if (row0 < rows) {
#pragma unroll
        for (int j = 0; j < kHeadCols / 8; ++j) {
            *reinterpret_cast<uint32_t*>(os + (row0 + gq) * ldo + j * 8 + 2 * tq) = pack_pair(acc[j][0], acc[j][1]);
            *reinterpret_cast<uint32_t*>(os + (row0 + gq + 8) * ldo + j * 8 + 2 * tq) = pack_pair(acc[j][2], acc[j][3]);
        }
    }
    __syncthreads();
    const int pieces = cols / 8;
    for (int i = threadIdx.x; i < rows * pieces; i += kRunThreads) {
        const int r = i / pieces, c = (i % pieces) * 8;
        *reinterpret_cast<uint4*>(out + (size_t)r * p.ldc + c) = *reinterpret_cast<const uint4*>(os + r * ldo + c);
    }
}

}  // namespace b200

// A, W and C bfloat16; k a multiple of 8, A's rows and W on 16-byte boundaries; kErrUnsupportedSize for operands it does not take.
extern "C" int b200_gemm_heads(const void* a, int lda, const void* w, void* c, int ldc, int M, int n, int k, int heads, cudaStream_t stream) {
    using namespace b200;
    if (M <= 0 || n <= 0 || heads <= 0) return 0;
    if (k < 8 || k % 8 != 0 || lda % 8 != 0 || (((uintptr_t)a | (uintptr_t)w) & 15)) return kErrUnsupportedSize;
    const long long ny = (n + kHeadCols - 1) / kHeadCols;
    if (heads > 65535 || ny > 65535) return kErrUnsupportedSize;
    const int ld = (k + 15) / 16 * 16 + 8;
    size_t smem = sizeof(__nv_bfloat16) * (size_t)(kRun + kHeadCols) * ld;
    const size_t results = sizeof(__nv_bfloat16) * (size_t)kRun * (kHeadCols + 8);
    if (smem < results) smem = results;
    if (smem > 226 * 1024) return kErrUnsupportedSize;
    static size_t have = 48 * 1024;
    if (smem > have) {
        const int e = (int)cudaFuncSetAttribute(gemm_heads_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != 0) return e;
        have = smem;
    }
    const HeadProductArgs p = {(const __nv_bfloat16*)a, (const __nv_bfloat16*)w, (__nv_bfloat16*)c, lda, ldc, M, n, k,
                               n % 8 == 0 && ldc % 8 == 0 && ((uintptr_t)c & 15) == 0};
    return launch_pdl(gemm_heads_kernel, dim3((M + kRun - 1) / kRun, (unsigned)ny, heads), dim3(kRunThreads), smem, stream, p);
}
