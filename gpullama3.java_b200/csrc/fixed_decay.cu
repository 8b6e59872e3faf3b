// Linear attention whose state decays by a fixed factor per head (retention, lightning attention):
//     S_t = g S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t           per sequence and head; S [d_k, d_v] in 32 bits, in its cache slot
// with q, k and v the projections' rows, optionally passed through SiLU, q and k optionally turned by the token's position
// over halves of their first 2 `pairs` numbers, q multiplied by a scale.  All of that is 32-bit.
//
// One token per sequence (fixed_decay_step): a CTA takes a head's columns of one sequence.  The state does not depend on the
// kernels before it in the step, so its first rows are on their way before the dependency wait, as are the angles.  Where
// the CTA has all columns of its head it can finish the head too: o / rms(o), times the output gate.
//
// Many tokens (bfloat16 operands): because g is a constant, a run of kRun tokens can be taken at once.  With tokens numbered
// i = 0 .. n - 1 inside a run and S the state before it,
//     o_i = sum_(j <= i) g^(i - j) (q_i . k_j) v_j + g^(i + 1) S^T q_i          S' = g^n S + sum_j g^(n - 1 - j) k_j v_j^T
// so the work is (1) every run's own sum of outer products, all runs of all heads at once, (2) the states before every
// run, a short sequential pass over the runs' sums, element by element, (3) the outputs, all runs of all heads at once.
// (1) and (3) are products of 64-token tiles on the tensor cores.  What enters the recurrence is kept in 32 bits, and a
// tensor-core operand has 16: q, k, the decayed keys, the decayed scores and the state therefore enter as the sum of two
// bfloat16 numbers (x = hi + lo, 16 bits of mantissa), products of two such sums without the lo lo term; sums are 32-bit.
// The powers of g are exact to 32-bit rounding (powf).  v enters as one bfloat16 number (it is a projection with its activation).
// A sequence's runs start at the step's first token of the sequence; the last one may be short.
#include "common.cuh"

namespace b200 {

constexpr int kRun = 64;          // tokens of a run
constexpr int kRunThreads = 128;  // four warps of 16 token rows

struct FixedDecayArgs {
    const void* q;          // [T, ld_qk], head h at column h d_k
    const void* k;
    const void* v;          // [T, ld_v], head h at column h d_v
    int ld_q, ld_k, ld_v;
    const float* decay;     // [heads]
    float* state;           // per slot: [heads][d_k][d_v]
    size_t slot_stride;
    const int* slots;
    const int* cu_seqlens;
    const float* inv_freq;  // [pairs] or null
    const int* positions;   // [T]
    const float2* angles;   // [pairs][T] (cos, sin) or null: the prompt kernels read these
    float* out;             // [T, heads d_v] 32-bit, or null when the head is finished here
    float* runs;            // scratch of the prompt kernels: [run][head][d_k][d_v]
    int n_tokens, heads, d_k, d_v, pairs, qk_silu, v_silu;
    float q_scale;
    // the finished head: o / sqrt(mean(o^2) + eps) * act(gate) * mul into columns of a buffer of the operands' type
    const void* gate;       // [T, ld_gate], head h at column h d_v
    int ld_gate, gate_act;  // 0 sigmoid, 1 SiLU
    void* rows;             // [T, ld_rows]
    int ld_rows;
    float eps, mul;
};

__device__ __forceinline__ float silu_32(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float gate_32(float z, int act) {
    const float s = 1.0f / (1.0f + expf(-z));
    return act == 1 ? z * s : s;
}

// ---------------------------------------------------------------------------------------------
// One token per sequence.  A row of the state is shared by TPR threads of VEC columns each; the CTA's eight groups of TPR
// threads take rows g, g + 8, ... and their partial read-outs meet in shared memory in the order of the groups.
constexpr int kStepGroups = 8, kStepRows = 8;   // rows per thread in flight: 64 rows of the state per round

template <typename T, int VEC, int TPR>
__global__ void __launch_bounds__(kStepGroups * TPR)
fixed_decay_step_kernel(FixedDecayArgs a) {
    constexpr int COLS = VEC * TPR, THREADS = kStepGroups * TPR;
    extern __shared__ float smem[];
    float* q_s = smem;                  // [d_k]
    float* k_s = q_s + a.d_k;           // [d_k]
    float* part = k_s + a.d_k;          // [groups][COLS]
    float* turn = part + kStepGroups * COLS;    // [pairs] cos, [pairs] sin
    __shared__ float scratch[33];
    const int h = blockIdx.y, t = blockIdx.z, col0 = blockIdx.x * COLS;
    const int tid = threadIdx.x, group = tid / TPR, lane_col = tid % TPR, col = col0 + lane_col * VEC;
    const bool live = col < a.d_v;
    pdl_launch_dependents();
    // (slots, positions and the state were written before the step's first kernel)
    float* S = a.state + (size_t)a.slots[t] * a.slot_stride + (size_t)h * a.d_k * a.d_v + col;
    float s[kStepRows][VEC];
    auto load_rows = [&](int base) {
#pragma unroll
        for (int i = 0; i < kStepRows; ++i) {
            const int r = base + i * kStepGroups + group;
            const bool ok = live && r < a.d_k;
            if constexpr (VEC == 4) {
                const float4 x = ok ? *reinterpret_cast<const float4*>(S + (size_t)r * a.d_v) : make_float4(0.f, 0.f, 0.f, 0.f);
                s[i][0] = x.x; s[i][1] = x.y; s[i][2] = x.z; s[i][3] = x.w;
            } else {
                s[i][0] = ok ? S[(size_t)r * a.d_v] : 0.f;
            }
        }
    };
    load_rows(0);
    const float g = a.decay[h];
    if (a.pairs > 0) {
        const float pos = (float)a.positions[t];
        for (int i = tid; i < a.pairs; i += THREADS) sincosf(pos * a.inv_freq[i], &turn[a.pairs + i], &turn[i]);
        __syncthreads();
    }
    pdl_wait();
    const T* qr = (const T*)a.q + (size_t)t * a.ld_q + (size_t)h * a.d_k;
    const T* kr = (const T*)a.k + (size_t)t * a.ld_k + (size_t)h * a.d_k;
    for (int i = tid; i < a.d_k; i += THREADS) {
        float qv = to_f32<T>(qr[i]), kv = to_f32<T>(kr[i]);
        if (a.qk_silu) { qv = silu_32(qv); kv = silu_32(kv); }
        if (i < 2 * a.pairs) {
            const bool first = i < a.pairs;
            const int other = first ? i + a.pairs : i - a.pairs, p = first ? i : other;
            float qo = to_f32<T>(qr[other]), ko = to_f32<T>(kr[other]);
            if (a.qk_silu) { qo = silu_32(qo); ko = silu_32(ko); }
            const float cs = turn[p], sn = first ? -turn[a.pairs + p] : turn[a.pairs + p];
            qv = qv * cs + qo * sn;
            kv = kv * cs + ko * sn;
        }
        q_s[i] = qv * a.q_scale;
        k_s[i] = kv;
    }
    float v[VEC], o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        v[e] = live ? to_f32<T>(((const T*)a.v)[(size_t)t * a.ld_v + (size_t)h * a.d_v + col + e]) : 0.f;
        if (a.v_silu) v[e] = silu_32(v[e]);
        o[e] = 0.f;
    }
    __syncthreads();
    for (int base = 0; base < a.d_k; base += kStepGroups * kStepRows) {
        if (base > 0) load_rows(base);
#pragma unroll
        for (int i = 0; i < kStepRows; ++i) {
            const int r = base + i * kStepGroups + group;
            if (r < a.d_k) {
                const float kk = k_s[r], qq = q_s[r];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[i][e] = g * s[i][e] + kk * v[e];
                    o[e] += qq * s[i][e];
                }
                if (live) {
                    if constexpr (VEC == 4) *reinterpret_cast<float4*>(S + (size_t)r * a.d_v) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
                    else S[(size_t)r * a.d_v] = s[i][0];
                }
            }
        }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) part[group * COLS + lane_col * VEC + e] = o[e];
    __syncthreads();
    float mine = 0.f;
    const int c = tid;       // (COLS <= THREADS)
    const bool owns = c < COLS && col0 + c < a.d_v;
    if (owns) {
#pragma unroll
        for (int w = 0; w < kStepGroups; ++w) mine += part[w * COLS + c];
    }
    if (a.rows == nullptr) {
        if (owns) a.out[((size_t)t * a.heads + h) * a.d_v + col0 + c] = mine;
        return;
    }
    const float ss = block_sum(owns ? mine * mine : 0.f, scratch);
    if (owns) {
        const float gate = gate_32(to_f32<T>(((const T*)a.gate)[(size_t)t * a.ld_gate + (size_t)h * a.d_v + c]), a.gate_act);
        ((T*)a.rows)[(size_t)t * a.ld_rows + (size_t)h * a.d_v + c] = from_f32<T>(mine * (a.mul / sqrtf(ss / (float)a.d_v + a.eps)) * gate);
    }
}

// ---------------------------------------------------------------------------------------------
// Many tokens.
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
// x = hi + lo in two bfloat16 numbers
__device__ __forceinline__ void split_store(__nv_bfloat16* hi, __nv_bfloat16* lo, float x) {
    const __nv_bfloat16 h = __float2bfloat16_rn(x);
    *hi = h;
    *lo = __float2bfloat16_rn(x - __bfloat162float(h));
}
__device__ __forceinline__ void split_store8(__nv_bfloat16* hi, __nv_bfloat16* lo, const float (&x)[8]) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float a = x[2 * i], b = x[2 * i + 1];
        h[i] = pack_pair(a, b);
        l[i] = pack_pair(a - __uint_as_float(h[i] << 16), b - __uint_as_float(h[i] & 0xffff0000u));
    }
    *reinterpret_cast<uint4*>(hi) = make_uint4(h[0], h[1], h[2], h[3]);
    *reinterpret_cast<uint4*>(lo) = make_uint4(l[0], l[1], l[2], l[3]);
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

// A run's rows of q or k as hi and lo tiles [kRun][ld] in shared memory (columns d_k .. d_pad and rows beyond the run
// zero), each row times factor[row] (null: 1) and `scale`.  Two threads share a token's row; 8 numbers per access where the
// rows lie on 16-byte boundaries.
__device__ __forceinline__ void load_rows_split(const FixedDecayArgs& a, const __nv_bfloat16* src, int ld_src, int first, int n, int h,
                                                __nv_bfloat16* hi, __nv_bfloat16* lo, int ld, int d_pad, float scale,
                                                const float* factor) {
    const int r = threadIdx.x & (kRun - 1), part = threadIdx.x >> 6;
    __nv_bfloat16* hr = hi + (size_t)r * ld;
    __nv_bfloat16* lr = lo + (size_t)r * ld;
    if (r >= n) {
        for (int c = part * 8; c < d_pad; c += 16) {
            *reinterpret_cast<uint4*>(hr + c) = make_uint4(0, 0, 0, 0);
            *reinterpret_cast<uint4*>(lr + c) = make_uint4(0, 0, 0, 0);
        }
        return;
    }
    const size_t t = (size_t)first + r;
    const __nv_bfloat16* x = src + t * ld_src + (size_t)h * a.d_k;
    const float f = scale * (factor ? factor[r] : 1.f);
    const float2* ang = a.angles + t;
    const size_t T = (size_t)a.n_tokens;
    const bool vec = a.d_k % 8 == 0 && a.pairs % 8 == 0 && ld_src % 8 == 0 && ((uintptr_t)src & 15) == 0;
    if (vec) {
        for (int c = part * 8; c < a.pairs; c += 16) {
            float u[8], v[8];
            load8(x + c, u);
            load8(x + a.pairs + c, v);
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                if (a.qk_silu) { u[e] = silu_32(u[e]); v[e] = silu_32(v[e]); }
                const float2 cs = ang[(size_t)(c + e) * T];
                const float p = u[e] * cs.x - v[e] * cs.y, q = v[e] * cs.x + u[e] * cs.y;
                u[e] = p * f;
                v[e] = q * f;
            }
            split_store8(hr + c, lr + c, u);
            split_store8(hr + a.pairs + c, lr + a.pairs + c, v);
        }
        for (int c = 2 * a.pairs + part * 8; c < a.d_k; c += 16) {
            float u[8];
            load8(x + c, u);
#pragma unroll
            for (int e = 0; e < 8; ++e) u[e] = (a.qk_silu ? silu_32(u[e]) : u[e]) * f;
            split_store8(hr + c, lr + c, u);
        }
    } else {
        for (int c = part; c < a.pairs; c += 2) {
            float u = __bfloat162float(x[c]), v = __bfloat162float(x[c + a.pairs]);
            if (a.qk_silu) { u = silu_32(u); v = silu_32(v); }
            const float2 cs = ang[(size_t)c * T];
            split_store(hr + c, lr + c, (u * cs.x - v * cs.y) * f);
            split_store(hr + c + a.pairs, lr + c + a.pairs, (v * cs.x + u * cs.y) * f);
        }
        for (int c = 2 * a.pairs + part; c < a.d_k; c += 2) {
            const float u = __bfloat162float(x[c]);
            split_store(hr + c, lr + c, (a.qk_silu ? silu_32(u) : u) * f);
        }
    }
    for (int c = a.d_k + part; c < d_pad; c += 2) {
        hr[c] = __float2bfloat16_rn(0.f);
        lr[c] = __float2bfloat16_rn(0.f);
    }
}

// columns col0 .. col0 + NS of the run's values as one tile [kRun][ld]
template <int NS>
__device__ __forceinline__ void load_values(const FixedDecayArgs& a, int first, int n, int h, int col0, __nv_bfloat16* dst, int ld) {
    const __nv_bfloat16* src = (const __nv_bfloat16*)a.v;
    const bool vec = a.d_v % 8 == 0 && a.ld_v % 8 == 0 && ((uintptr_t)src & 15) == 0;
    for (int i = threadIdx.x; i < kRun * (NS / 8); i += kRunThreads) {
        const int r = i / (NS / 8), c = (i % (NS / 8)) * 8;
        __nv_bfloat16* o = dst + (size_t)r * ld + c;
        const __nv_bfloat16* x = src + ((size_t)first + r) * a.ld_v + (size_t)h * a.d_v + col0 + c;
        if (r >= n || col0 + c >= a.d_v) {
            *reinterpret_cast<uint4*>(o) = make_uint4(0, 0, 0, 0);
        } else if (vec) {
            if (a.v_silu) {
                float f[8];
                load8(x, f);
                *reinterpret_cast<uint4*>(o) = make_uint4(pack_pair(silu_32(f[0]), silu_32(f[1])), pack_pair(silu_32(f[2]), silu_32(f[3])),
                                                         pack_pair(silu_32(f[4]), silu_32(f[5])), pack_pair(silu_32(f[6]), silu_32(f[7])));
            } else {
                *reinterpret_cast<uint4*>(o) = *reinterpret_cast<const uint4*>(x);
            }
        } else {
            for (int e = 0; e < 8; ++e) {
                const float f = col0 + c + e < a.d_v ? __bfloat162float(x[e]) : 0.f;
                o[e] = __float2bfloat16_rn(a.v_silu ? silu_32(f) : f);
            }
        }
    }
}

// where a sequence's runs start in the scratch: a bound on the runs of the sequences before it that needs no sum over them
__device__ __forceinline__ int first_run(const int* cu_seqlens, int seq) { return cu_seqlens[seq] / kRun + seq; }

// powers g^0 .. g^kRun in shared memory
__device__ __forceinline__ void powers(float* pw, float g) {
    for (int i = threadIdx.x; i <= kRun; i += kRunThreads) pw[i] = i == 0 ? 1.f : powf(g, (float)i);
}

// (1) U[d_k, columns] = sum_j g^(n - 1 - j) k_j v_j^T of one run
template <int NS>
__global__ void __launch_bounds__(kRunThreads)
fixed_decay_run_sums_kernel(FixedDecayArgs a) {
    extern __shared__ __align__(16) uint8_t run_smem[];
    const int slices = (a.d_v + NS - 1) / NS;
    const int run = blockIdx.x / slices, col0 = (blockIdx.x % slices) * NS, h = blockIdx.y, seq = blockIdx.z;
    const int seq0 = a.cu_seqlens[seq], q_len = a.cu_seqlens[seq + 1] - seq0;
    pdl_launch_dependents();
    const int d_pad = (a.d_k + 15) / 16 * 16, ld = d_pad + 8, ldv = NS + 8;
    __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(run_smem);
    __nv_bfloat16* klo = khi + kRun * ld;
    __nv_bfloat16* vs = klo + kRun * ld;
    __shared__ float pw[kRun + 1], factor[kRun];
    powers(pw, a.decay[h]);
    __syncthreads();
    const int first = seq0 + run * kRun, n = min(kRun, q_len - run * kRun);
    if (threadIdx.x < kRun) factor[threadIdx.x] = (int)threadIdx.x < n ? pw[n - 1 - threadIdx.x] : 0.f;
    __syncthreads();
    pdl_wait();
    if (n <= 0) return;
    load_rows_split(a, (const __nv_bfloat16*)a.k, a.ld_k, first, n, h, khi, klo, ld, d_pad, 1.f, factor);
    load_values<NS>(a, first, n, h, col0, vs, ldv);
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3, mr = lane & 7, gq = lane >> 2, tq = lane & 3;
    float* U = a.runs + ((size_t)(first_run(a.cu_seqlens, seq) + run) * a.heads + h) * a.d_k * a.d_v;
    for (int m = warp; m < d_pad / 16; m += kRunThreads / 32) {
        float acc[NS / 8][4];
#pragma unroll
        for (int j = 0; j < NS / 8; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
#pragma unroll
        for (int kk = 0; kk < kRun / 16; ++kk) {
            if (kk * 16 >= n) break;
            // A = the decayed keys transposed: token rows in shared memory, so the transposing load
            uint32_t ah[4], al[4];
            const int at = (kk * 16 + (mi >> 1) * 8 + mr) * ld + m * 16 + (mi & 1) * 8;
            ldsm4t(ah, khi + at);
            ldsm4t(al, klo + at);
#pragma unroll
            for (int j = 0; j < NS / 16; ++j) {
                uint32_t b[4];
                ldsm4t(b, vs + (kk * 16 + (mi & 1) * 8 + mr) * ldv + j * 16 + (mi >> 1) * 8);
                mma_run(acc[2 * j], ah, b[0], b[1]);
                mma_run(acc[2 * j], al, b[0], b[1]);
                mma_run(acc[2 * j + 1], ah, b[2], b[3]);
                mma_run(acc[2 * j + 1], al, b[2], b[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < NS / 8; ++j) {
            const int c = col0 + j * 8 + 2 * tq;
#pragma unroll
            for (int hh = 0; hh < 2; ++hh) {
                const int r = m * 16 + gq + 8 * hh;
                if (r >= a.d_k) continue;
                float* u = U + (size_t)r * a.d_v + c;
                if (c + 1 < a.d_v && a.d_v % 2 == 0) *reinterpret_cast<float2*>(u) = make_float2(acc[j][2 * hh], acc[j][2 * hh + 1]);
                else {
                    if (c < a.d_v) u[0] = acc[j][2 * hh];
                    if (c + 1 < a.d_v) u[1] = acc[j][2 * hh + 1];
                }
            }
        }
    }
}

// (2) per element, run after run: the scratch's run sum is replaced by the state before the run; the state after the last
// run goes back to the slot.  Eight runs' sums are asked for at once.
__global__ void __launch_bounds__(256)
fixed_decay_carry_kernel(FixedDecayArgs a) {
    const int h = blockIdx.y, seq = blockIdx.z;
    const int per_head = a.d_k * a.d_v, e = blockIdx.x * 256 + threadIdx.x;
    const int q_len = a.cu_seqlens[seq + 1] - a.cu_seqlens[seq];
    const int n_runs = (q_len + kRun - 1) / kRun;
    pdl_launch_dependents();
    const float g = a.decay[h], g_run = powf(g, (float)kRun), g_last = powf(g, (float)(q_len - (n_runs - 1) * kRun));
    pdl_wait();
    if (e >= per_head || n_runs == 0) return;
    float* S = a.state + (size_t)a.slots[seq] * a.slot_stride + (size_t)h * per_head + e;
    float carry = *S;
    const size_t step = (size_t)a.heads * per_head;
    float* u = a.runs + ((size_t)first_run(a.cu_seqlens, seq) * a.heads + h) * per_head + e;
    for (int r0 = 0; r0 < n_runs; r0 += 8) {
        float x[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = r0 + i < n_runs ? u[(size_t)(r0 + i) * step] : 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (r0 + i < n_runs) {
                u[(size_t)(r0 + i) * step] = carry;
                carry = (r0 + i == n_runs - 1 ? g_last : g_run) * carry + x[i];
            }
        }
    }
    *S = carry;
}

// (3) outputs of one run
template <int NS>
__global__ void __launch_bounds__(kRunThreads)
fixed_decay_outputs_kernel(FixedDecayArgs a) {
    extern __shared__ __align__(16) uint8_t run_smem[];
    const int slices = (a.d_v + NS - 1) / NS;
    const int run = blockIdx.x / slices, col0 = (blockIdx.x % slices) * NS, h = blockIdx.y, seq = blockIdx.z;
    const int seq0 = a.cu_seqlens[seq], q_len = a.cu_seqlens[seq + 1] - seq0;
    pdl_launch_dependents();
    const int d_pad = (a.d_k + 15) / 16 * 16, ld = d_pad + 8, ldv = NS + 8;
    __nv_bfloat16* qhi = reinterpret_cast<__nv_bfloat16*>(run_smem);
    __nv_bfloat16* qlo = qhi + kRun * ld;
    __nv_bfloat16* khi = qlo + kRun * ld;
    __nv_bfloat16* klo = khi + kRun * ld;
    __nv_bfloat16* vs = klo + kRun * ld;
    __nv_bfloat16* shi = vs + kRun * ldv;
    __nv_bfloat16* slo = shi + d_pad * ldv;
    __shared__ float pw[kRun + 1];
    powers(pw, a.decay[h]);
    const int first = seq0 + run * kRun, n = min(kRun, q_len - run * kRun);
    pdl_wait();
    if (n <= 0) return;
    load_rows_split(a, (const __nv_bfloat16*)a.q, a.ld_q, first, n, h, qhi, qlo, ld, d_pad, a.q_scale, nullptr);
    load_rows_split(a, (const __nv_bfloat16*)a.k, a.ld_k, first, n, h, khi, klo, ld, d_pad, 1.f, nullptr);
    load_values<NS>(a, first, n, h, col0, vs, ldv);
    {   // the state before the run: 8 numbers per thread and access where the rows allow it
        const float* S = a.runs + ((size_t)(first_run(a.cu_seqlens, seq) + run) * a.heads + h) * a.d_k * a.d_v;
        const bool vec = a.d_v % 8 == 0 && ((uintptr_t)a.runs & 15) == 0;
        for (int i = threadIdx.x; i < d_pad * (NS / 8); i += kRunThreads) {
            const int r = i / (NS / 8), c = (i % (NS / 8)) * 8;
            float x[8];
            if (r < a.d_k && col0 + c + 8 <= a.d_v && vec) {
                const float4* p = reinterpret_cast<const float4*>(S + (size_t)r * a.d_v + col0 + c);
                const float4 u = p[0], v = p[1];
                x[0] = u.x; x[1] = u.y; x[2] = u.z; x[3] = u.w; x[4] = v.x; x[5] = v.y; x[6] = v.z; x[7] = v.w;
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] = (r < a.d_k && col0 + c + e < a.d_v) ? S[(size_t)r * a.d_v + col0 + c + e] : 0.f;
            }
            split_store8(shi + (size_t)r * ldv + c, slo + (size_t)r * ldv + c, x);
        }
    }
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3, mr = lane & 7, gq = lane >> 2, tq = lane & 3;
    const int row0 = warp * 16;
    if (row0 >= n) return;      // (no barrier below)
    float o[NS / 8][4], sc[kRun / 8][4];
#pragma unroll
    for (int j = 0; j < NS / 8; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[j][i] = 0.f;
#pragma unroll
    for (int j = 0; j < kRun / 8; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) sc[j][i] = 0.f;
    // scores against the run's tokens up to this warp's last row, and the read-out of the state before the run
    for (int kk = 0; kk < d_pad / 16; ++kk) {
        uint32_t ah[4], al[4];
        const int at = (row0 + (mi & 1) * 8 + mr) * ld + kk * 16 + (mi >> 1) * 8;
        ldsm4(ah, qhi + at);
        ldsm4(al, qlo + at);
#pragma unroll
        for (int j = 0; j < kRun / 16; ++j) {
            if (j <= warp) {
                uint32_t bh[4], bl[4];
                const int bt = (j * 16 + (mi >> 1) * 8 + mr) * ld + kk * 16 + (mi & 1) * 8;
                ldsm4(bh, khi + bt);
                ldsm4(bl, klo + bt);
                mma_run(sc[2 * j], ah, bh[0], bh[1]);
                mma_run(sc[2 * j], ah, bl[0], bl[1]);
                mma_run(sc[2 * j], al, bh[0], bh[1]);
                mma_run(sc[2 * j + 1], ah, bh[2], bh[3]);
                mma_run(sc[2 * j + 1], ah, bl[2], bl[3]);
                mma_run(sc[2 * j + 1], al, bh[2], bh[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < NS / 16; ++j) {
            uint32_t bh[4], bl[4];
            const int bt = (kk * 16 + (mi & 1) * 8 + mr) * ldv + j * 16 + (mi >> 1) * 8;
            ldsm4t(bh, shi + bt);
            ldsm4t(bl, slo + bt);
            mma_run(o[2 * j], ah, bh[0], bh[1]);
            mma_run(o[2 * j], ah, bl[0], bl[1]);
            mma_run(o[2 * j], al, bh[0], bh[1]);
            mma_run(o[2 * j + 1], ah, bh[2], bh[3]);
            mma_run(o[2 * j + 1], ah, bl[2], bl[3]);
            mma_run(o[2 * j + 1], al, bh[2], bh[3]);
        }
    }
    const int i0 = row0 + gq, i1 = i0 + 8;
    const float f0 = pw[i0 + 1], f1 = pw[i1 + 1];
#pragma unroll
    for (int j = 0; j < NS / 8; ++j) {
        o[j][0] *= f0; o[j][1] *= f0;
        o[j][2] *= f1; o[j][3] *= f1;
    }
    // the decayed scores times the run's values
#pragma unroll
    for (int j = 0; j < kRun / 16; ++j) {
        if (j > warp) continue;
        uint32_t ah[4], al[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int c = j * 16 + half * 8 + 2 * tq;
            float p[4];
            p[0] = c <= i0 ? sc[2 * j + half][0] * pw[max(i0 - c, 0)] : 0.f;
            p[1] = c + 1 <= i0 ? sc[2 * j + half][1] * pw[max(i0 - c - 1, 0)] : 0.f;
            p[2] = c <= i1 ? sc[2 * j + half][2] * pw[max(i1 - c, 0)] : 0.f;
            p[3] = c + 1 <= i1 ? sc[2 * j + half][3] * pw[max(i1 - c - 1, 0)] : 0.f;
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const uint32_t hi = pack_pair(p[2 * r], p[2 * r + 1]);
                ah[2 * half + r] = hi;
                al[2 * half + r] = pack_pair(p[2 * r] - __uint_as_float(hi << 16), p[2 * r + 1] - __uint_as_float(hi & 0xffff0000u));
            }
        }
#pragma unroll
        for (int jj = 0; jj < NS / 16; ++jj) {
            uint32_t b[4];
            ldsm4t(b, vs + (j * 16 + (mi & 1) * 8 + mr) * ldv + jj * 16 + (mi >> 1) * 8);
            mma_run(o[2 * jj], ah, b[0], b[1]);
            mma_run(o[2 * jj], al, b[0], b[1]);
            mma_run(o[2 * jj + 1], ah, b[2], b[3]);
            mma_run(o[2 * jj + 1], al, b[2], b[3]);
        }
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        const int i = hh ? i1 : i0;
        if (a.rows != nullptr) {
            // the head is finished here: its numbers lie in the four lanes of the row (columns beyond d_v are zero)
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < NS / 8; ++j) ss += o[j][2 * hh] * o[j][2 * hh] + o[j][2 * hh + 1] * o[j][2 * hh + 1];
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            if (i >= n) continue;
            const float scale = a.mul / sqrtf(ss / (float)a.d_v + a.eps);
            const size_t t = (size_t)first + i;
            const __nv_bfloat16* gate = (const __nv_bfloat16*)a.gate + t * a.ld_gate + (size_t)h * a.d_v;
            __nv_bfloat16* dst = (__nv_bfloat16*)a.rows + t * a.ld_rows + (size_t)h * a.d_v;
            const bool pairs = (((uintptr_t)gate | (uintptr_t)dst) & 3) == 0;
#pragma unroll
            for (int j = 0; j < NS / 8; ++j) {
                const int c = j * 8 + 2 * tq;
                if (c + 1 < a.d_v && pairs) {
                    const uint32_t g2 = *reinterpret_cast<const uint32_t*>(gate + c);
                    *reinterpret_cast<uint32_t*>(dst + c) =
                        pack_pair(o[j][2 * hh] * scale * gate_32(__uint_as_float(g2 << 16), a.gate_act),
                                  o[j][2 * hh + 1] * scale * gate_32(__uint_as_float(g2 & 0xffff0000u), a.gate_act));
                } else {
                    for (int e = 0; e < 2; ++e)
                        if (c + e < a.d_v)
                            dst[c + e] = __float2bfloat16_rn(o[j][2 * hh + e] * scale * gate_32(__bfloat162float(gate[c + e]), a.gate_act));
                }
            }
        } else {
            if (i >= n) continue;
            float* dst = a.out + (((size_t)first + i) * a.heads + h) * a.d_v + col0;
#pragma unroll
            for (int j = 0; j < NS / 8; ++j) {
                const int c = j * 8 + 2 * tq;
                if (col0 + c + 1 < a.d_v && a.d_v % 2 == 0) *reinterpret_cast<float2*>(dst + c) = make_float2(o[j][2 * hh], o[j][2 * hh + 1]);
                else {
                    if (col0 + c < a.d_v) dst[c] = o[j][2 * hh];
                    if (col0 + c + 1 < a.d_v) dst[c + 1] = o[j][2 * hh + 1];
                }
            }
        }
    }
}

static size_t outputs_smem(int d_k, int ns) {
    const int d_pad = (d_k + 15) / 16 * 16;
    return sizeof(__nv_bfloat16) * ((size_t)4 * kRun * (d_pad + 8) + (size_t)kRun * (ns + 8) + (size_t)2 * d_pad * (ns + 8));
}
static size_t sums_smem(int d_k, int ns) {
    const int d_pad = (d_k + 15) / 16 * 16;
    return sizeof(__nv_bfloat16) * ((size_t)2 * kRun * (d_pad + 8) + (size_t)kRun * (ns + 8));
}
constexpr size_t kMostSmem = 227 * 1024 - 1024;    // (a kilobyte for the static part)

// columns of the values a CTA takes: all of a head's up to 128 where shared memory allows, else slices of 64; 0: no fit
static int run_columns(int d_k, int d_v) {
    if (d_v > 64 && outputs_smem(d_k, 128) <= kMostSmem) return 128;
    return outputs_smem(d_k, 64) <= kMostSmem ? 64 : 0;
}

template <int NS>
static int launch_runs(const FixedDecayArgs& a, int n_seqs, int max_q_len, cudaStream_t stream) {
    const size_t s1 = sums_smem(a.d_k, NS), s3 = outputs_smem(a.d_k, NS);
    static size_t have1 = 48 * 1024, have3 = 48 * 1024;
    if (s1 > have1) {
        const int e = (int)cudaFuncSetAttribute(fixed_decay_run_sums_kernel<NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        if (e != 0) return e;
        have1 = s1;
    }
    if (s3 > have3) {
        const int e = (int)cudaFuncSetAttribute(fixed_decay_outputs_kernel<NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
        if (e != 0) return e;
        have3 = s3;
    }
    const int n_runs = (max_q_len + kRun - 1) / kRun, slices = (a.d_v + NS - 1) / NS;
    const dim3 grid(n_runs * slices, a.heads, n_seqs);
    int st = launch_pdl(fixed_decay_run_sums_kernel<NS>, grid, dim3(kRunThreads), s1, stream, a);
    if (st != 0) return st;
    st = launch_pdl(fixed_decay_carry_kernel, dim3((a.d_k * a.d_v + 255) / 256, a.heads, n_seqs), dim3(256), 0, stream, a);
    if (st != 0) return st;
    return launch_pdl(fixed_decay_outputs_kernel<NS>, grid, dim3(kRunThreads), s3, stream, a);
}

template <typename T, int VEC, int TPR>
static int launch_step(const FixedDecayArgs& a, cudaStream_t stream) {
    constexpr int COLS = VEC * TPR;
    const size_t smem = sizeof(float) * ((size_t)2 * a.d_k + (size_t)kStepGroups * COLS + 2 * (size_t)a.pairs);
    const dim3 grid((a.d_v + COLS - 1) / COLS, a.heads, a.n_tokens);
    return launch_pdl(fixed_decay_step_kernel<T, VEC, TPR>, grid, dim3(kStepGroups * TPR), smem, stream, a);
}

}  // namespace b200

// Columns of a head's values that one CTA of the prompt kernels takes (0: they do not take this key size), and whether
// they, or the one-token kernel, can finish a head (all its values in one CTA).
extern "C" int b200_fixed_decay_columns(int d_k, int d_v) { return b200::run_columns(d_k, d_v); }
extern "C" int b200_fixed_decay_step_finishes(int d_v) { return d_v % 4 == 0 ? d_v <= 128 : d_v <= 32; }
// Runs the scratch of the prompt kernels has room for: n_runs * heads * d_k * d_v floats.
extern "C" int b200_fixed_decay_runs(int n_tokens, int n_seqs) { return n_tokens / b200::kRun + n_seqs + 1; }

// The recurrence over a packed step (see the head of this file).  n_tokens == n_seqs: one token per sequence, operands of
// either type; otherwise bfloat16 operands, `scratch` as b200_fixed_decay_runs says and `angles` [pairs][T] (cos, sin).
// out: float32 [T, heads d_v], or rows (not null): the finished heads, o / rms(o) * act(gate) * mul, into [T, ld_rows].
extern "C" int b200_fixed_decay(const void* q, int ld_q, const void* k, int ld_k, const void* v, int ld_v, const float* decay,
                                float* state, long long slot_stride, const int* slots, const int* cu_seqlens, const int* positions,
                                const float* inv_freq, const float* angles, int pairs, float* out, float* scratch, int dtype,
                                int n_tokens, int n_seqs, int max_q_len, int heads, int d_k, int d_v, float q_scale, int qk_silu,
                                int v_silu, const void* gate, int ld_gate, int gate_act, void* rows, int ld_rows, float eps, float mul,
                                cudaStream_t stream) {
    using namespace b200;
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (heads < 1 || heads > 65535 || n_seqs > 65535 || d_k < 1 || d_v < 1 || d_k > 512 || pairs < 0 || 2 * pairs > d_k || !decay)
        return kErrBadArgument;
    if ((rows == nullptr) == (out == nullptr) || (rows != nullptr && (!gate || ld_rows < heads * d_v || ld_gate < heads * d_v)))
        return kErrBadArgument;
    FixedDecayArgs a = {q, k, v, ld_q, ld_k, ld_v, decay, state, (size_t)slot_stride, slots, cu_seqlens, inv_freq, positions,
                        (const float2*)angles, out, scratch, n_tokens, heads, d_k, d_v, pairs, qk_silu, v_silu, q_scale, gate, ld_gate,
                        gate_act, rows, ld_rows, eps, mul};
    if (n_tokens == n_seqs) {
        if (pairs > 0 && (!inv_freq || !positions)) return kErrBadArgument;
        if (rows != nullptr && !b200_fixed_decay_step_finishes(d_v)) return kErrUnsupportedSize;
        const bool vec = d_v % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
        if (rows != nullptr && !vec && d_v > 32) return kErrUnsupportedSize;
        B200_DISPATCH_DTYPE(dtype, T,
            if (!vec) return launch_step<T, 1, 32>(a, stream);
            if (d_v <= 64) return launch_step<T, 4, 16>(a, stream);
            return launch_step<T, 4, 32>(a, stream));
        return 0;
    }
    if (dtype != kBF16) return kErrUnsupportedSize;
    const int ns = run_columns(d_k, d_v);
    if (ns == 0) return kErrUnsupportedSize;
    if (rows != nullptr && d_v > ns) return kErrUnsupportedSize;
    if (!scratch || ((uintptr_t)scratch & 15) || (pairs > 0 && !angles)) return kErrBadArgument;
    return ns == 128 ? launch_runs<128>(a, n_seqs, max_q_len, stream) : launch_runs<64>(a, n_seqs, max_q_len, stream);
}
