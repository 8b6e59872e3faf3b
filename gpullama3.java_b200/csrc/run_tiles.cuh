// What the kernels share that take a recurrence in runs of 64 tokens as products on the tensor cores (mma.sync m16n8k16 over
// tiles of bfloat16 rows in shared memory): the tiles' loads, the fragments, numbers split in two bfloat16 parts.
#pragma once
#include "common.cuh"

namespace b200 {

constexpr int kRun = 64;          // tokens of a run
constexpr int kRunThreads = 128;  // four warps of 16 token rows

__device__ __forceinline__ float silu_32(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float gate_32(float z, int act) {
    const float s = 1.0f / (1.0f + expf(-z));
    return act == 1 ? z * s : s;
}

// the same with the hardware's exponential and reciprocal (relative error about 1e-6), for results that are rounded to 16 bits
__device__ __forceinline__ float gate_16(float z, int act) {
    const float s = __fdividef(1.0f, 1.0f + __expf(-z));
    return act == 1 ? z * s : s;
}

__device__ __forceinline__ void mma_run(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const __nv_bfloat16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ uint32_t pack_pair(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
// a pair of numbers as bfloat16 pairs hi and lo, x = hi + lo
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_pair(a, b);
    lo = pack_pair(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        f[2 * i] = __uint_as_float(w[i] << 16);
        f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}

__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
}

__device__ __forceinline__ void copy_16(__nv_bfloat16* dst, const __nv_bfloat16* src, bool take) {
    const int n = take ? 16 : 0;      // (0: zeros are written)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void copies_done() {
    asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
}

// columns 0 .. width of a run's rows as a tile [kRun][ld] (rows beyond the run and columns beyond `limit` zero)
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, int ld_src, int n, int width, int limit) {
    const int per_row = width / 8;
    for (int i = threadIdx.x; i < kRun * per_row; i += kRunThreads) {
        const int r = i / per_row, c = (i % per_row) * 8;
        const bool take = r < n && c < limit;
        copy_16(dst + (size_t)r * ld + c, take ? src + (size_t)r * ld_src + c : src, take);
    }
}

// columns col0 .. col0 + NS of a state [d_k][d_v] kept as (hi, lo) pairs of bfloat16 (one 32-bit word per number) as two tiles [d_pad][ldv]
// of its hi and lo parts, zeros beyond its edges: four numbers per thread and access where the rows allow it, eight accesses of a thread
// on their way at once
template <int NS>
__device__ __forceinline__ void load_state_parts(__nv_bfloat16* shi, __nv_bfloat16* slo, int ldv, const uint32_t* S, int d_k, int d_v, int col0, int d_pad) {
    const bool vec = d_v % 4 == 0;
    const int total = d_pad * (NS / 4);
    for (int base = threadIdx.x; base < total; base += 8 * kRunThreads) {
        uint4 x[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = base + u * kRunThreads, r = i / (NS / 4), c = (i % (NS / 4)) * 4;
            x[u] = make_uint4(0, 0, 0, 0);
            if (i < total && r < d_k && col0 + c < d_v) {
                const uint32_t* p = S + (size_t)r * d_v + col0 + c;
                if (vec) {
                    x[u] = *reinterpret_cast<const uint4*>(p);
                } else {
                    x[u].x = p[0];
                    x[u].y = col0 + c + 1 < d_v ? p[1] : 0u;
                    x[u].z = col0 + c + 2 < d_v ? p[2] : 0u;
                    x[u].w = col0 + c + 3 < d_v ? p[3] : 0u;
                }
            }
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = base + u * kRunThreads, r = i / (NS / 4), c = (i % (NS / 4)) * 4;
            if (i < total) {
                *reinterpret_cast<uint2*>(shi + (size_t)r * ldv + c) = make_uint2(__byte_perm(x[u].x, x[u].y, 0x5410), __byte_perm(x[u].z, x[u].w, 0x5410));
                *reinterpret_cast<uint2*>(slo + (size_t)r * ldv + c) = make_uint2(__byte_perm(x[u].x, x[u].y, 0x7632), __byte_perm(x[u].z, x[u].w, 0x7632));
            }
        }
    }
}

// where a sequence's runs start in the scratch: a bound on the runs of the sequences before it that needs no sum over them
__device__ __forceinline__ int first_run(const int* cu_seqlens, int seq) { return cu_seqlens[seq] / kRun + seq; }

}  // namespace b200
