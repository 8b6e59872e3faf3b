// A matrix memory per head with an exponential input gate and a forget gate that every token computes (the memory of an mLSTM),
// kept in range by a running maximum.  With the logits z_i, z_f of a token and head (projections plus bias), c the gate cap:
//     i = c tanh(z_i / c),  f = log sigmoid(c tanh(z_f / c))                            (both are logarithms of gates)
//     m_t = max(f + m_(t-1), i)                                                         (m starts at zero)
//     S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k_t v_t^T,   n_t alike with k_t alone
//     o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)                             (q carries a scale)
// Per slot: S of every head [d_k][d_v], then n of every head, then m of every head, all in 32 bits.  n and m exist in `copies`
// copies, one for each slice of a head's columns that the one-token kernel's CTAs take, so that no CTA reads what another writes.
//
// One token per sequence (memory_step): a CTA takes a slice of a head's columns of one sequence; state rows, n and m are on
// their way before the dependency wait.  A CTA with all columns of its head can finish the head: o / rms(o), times a weight,
// times the output gate.
//
// Many tokens.  memory_gates makes the gates of all tokens and the running maximum: (a, b) with m -> max(m + a, b) compose like
// (a1 + a2, max(b1 + a2, b2)), so a warp takes 64 tokens and a CTA 2,048 of them at once.  It leaves, per head and token, f, i,
// m and F, the sum of f from the start of the token's run of 64 up to the token.  With tokens numbered inside a run, m_- the
// maximum and S, n the memory before it,
//     o_i ~ sum_(j <= i) e^(F_i - F_j + i_j - m_i) (q_i . k_j) v_j + e^(F_i + m_- - m_i) S^T q_i      (the read-out; n . q alike)
//     S'  = e^(F_n + m_- - m_n) S + sum_j e^(F_n - F_j + i_j - m_n) k_j v_j^T
// which is the scheme of the fixed decays with weights in place of powers: (1) every run's own sum of outer products, (2) the
// memories before the runs, element by element, (3) the outputs.  (1) and (3) are products of 64-token tiles on the tensor
// cores; weighted keys, weighted scores and the memory enter as the sum of two bfloat16 numbers, projections as the one they
// are stored as, sums and weights are 32-bit.
//
// Where those kernels do not take the operands (32-bit runs, keys too long for their tiles) the token-by-token scan of
// delta_rule.cu walks the same gates; memory_divide then forms the quotient.
#include "run_tiles.cuh"

namespace b200 {

constexpr float kMemoryFloor = 1e-6f;    // what joins the divisor

struct MemoryArgs {
    const void* q;          // [T, ld_q], head h at column h d_k
    const void* k;
    const void* v;          // [T, ld_v], head h at column h d_v
    int ld_q, ld_k, ld_v;
    const void* zi;         // [T, ld_zi], column h: the input gate's logit before its bias
    const void* zf;
    int ld_zi, ld_zf;
    const float* bias_i;    // [heads]
    const float* bias_f;
    float cap;
    float* state;
    size_t slot_stride;
    const int* slots;
    const int* cu_seqlens;
    float* out;             // [T, heads d_v] 32-bit, or null when the head is finished here
    float* gates;           // [4][heads][T]: F, i, m, f
    float* start_m;         // [n_seqs][heads]: m before the step
    float* runs;            // [run][head][per_run]: the run's sum (S, then n); after (2) the memory before the run: S as (hi, lo)
                            // pairs of bfloat16 in the place of each number, n as it is
    const __nv_bfloat16* qt;   // how the run kernels read the operands: rows on 16-byte boundaries, heads head_qk (head_v) apart
    const __nv_bfloat16* kt;
    const __nv_bfloat16* vt;
    int ld_qt, ld_kt, ld_vt, head_qk, head_v;
    int n_tokens, n_seqs, heads, d_k, d_v, copies;
    float q_scale;
    // the finished head: o / sqrt(mean(o^2) + eps) * weight * act(gate) into columns of a buffer of the operands' type
    const float* weight;    // [heads d_v] or null
    const void* gate;       // [T, ld_gate], head h at column h d_v
    int ld_gate, gate_act;
    void* rows;             // [T, ld_rows]
    int ld_rows;
    float eps;
};

__device__ __forceinline__ float* memory_n(const MemoryArgs& a, float* slot, int h, int copy) {
    return slot + (size_t)a.heads * a.d_k * a.d_v + ((size_t)h * a.copies + copy) * a.d_k;
}
__device__ __forceinline__ float* memory_m(const MemoryArgs& a, float* slot, int h, int copy) {
    return slot + (size_t)a.heads * a.d_k * (a.d_v + a.copies) + (size_t)h * a.copies + copy;
}
__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
    const float y = cap * tanhf(z / cap);
    return fminf(y, 0.f) - log1pf(expf(-fabsf(y)));      // log sigmoid(y)
}

// ---------------------------------------------------------------------------------------------
// One token per sequence.  A row of S is shared by TPR threads of VEC columns each; the CTA's eight groups of TPR threads take
// rows g, g + 8, ... and their partial read-outs meet in shared memory in the order of the groups.
constexpr int kStepGroups = 8, kStepRows = 8, kStepMostKeys = 512;

template <typename T, int VEC, int TPR>
__global__ void __launch_bounds__(kStepGroups * TPR)
memory_step_kernel(MemoryArgs a) {
    constexpr int COLS = VEC * TPR, THREADS = kStepGroups * TPR, KEYS = (kStepMostKeys + THREADS - 1) / THREADS;
    extern __shared__ float smem[];
    float* q_s = smem;                  // [d_k]
    float* k_s = q_s + a.d_k;           // [d_k]
    float* part = k_s + a.d_k;          // [groups][COLS]
    __shared__ float scratch[33];
    const int slice = blockIdx.x, h = blockIdx.y, t = blockIdx.z, col0 = slice * COLS;
    const int tid = threadIdx.x, group = tid / TPR, lane_col = tid % TPR, col = col0 + lane_col * VEC;
    const bool live = col < a.d_v;
    pdl_launch_dependents();
    // (slots and the state were written before the step's first kernel)
    float* slot = a.state + (size_t)a.slots[t] * a.slot_stride;
    float* S = slot + (size_t)h * a.d_k * a.d_v + col;
    float* n_g = memory_n(a, slot, h, slice);
    float* m_g = memory_m(a, slot, h, slice);
    float s[kStepRows][VEC], n[KEYS];
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
#pragma unroll
    for (int i = 0; i < KEYS; ++i) n[i] = tid + i * THREADS < a.d_k ? n_g[tid + i * THREADS] : 0.f;
    const float m_old = *m_g, b_i = a.bias_i[h], b_f = a.bias_f[h];
    pdl_wait();
    const float li = log_input_gate(to_f32<T>(((const T*)a.zi)[(size_t)t * a.ld_zi + h]) + b_i, a.cap);
    const float lf = log_forget_gate(to_f32<T>(((const T*)a.zf)[(size_t)t * a.ld_zf + h]) + b_f, a.cap);
    const float m = fmaxf(lf + m_old, li), keep = expf(lf + m_old - m), take = expf(li - m);
    const T* qr = (const T*)a.q + (size_t)t * a.ld_q + (size_t)h * a.d_k;
    const T* kr = (const T*)a.k + (size_t)t * a.ld_k + (size_t)h * a.d_k;
    float nq = 0.f;
#pragma unroll
    for (int i = 0; i < KEYS; ++i) {
        const int e = tid + i * THREADS;
        if (e < a.d_k) {
            const float qv = to_f32<T>(qr[e]) * a.q_scale, kv = to_f32<T>(kr[e]);
            q_s[e] = qv;
            k_s[e] = kv;
            n[i] = keep * n[i] + take * kv;
            nq += n[i] * qv;
        }
    }
    float v[VEC], o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        v[e] = live ? take * to_f32<T>(((const T*)a.v)[(size_t)t * a.ld_v + (size_t)h * a.d_v + col + e]) : 0.f;
        o[e] = 0.f;
    }
    nq = block_sum(nq, scratch);         // (its barriers stand between the writes of q_s, k_s and their reads, and behind every read of m)
#pragma unroll
    for (int i = 0; i < KEYS; ++i)
        if (tid + i * THREADS < a.d_k) n_g[tid + i * THREADS] = n[i];
    if (tid == 0) *m_g = m;
    for (int base = 0; base < a.d_k; base += kStepGroups * kStepRows) {
        if (base > 0) load_rows(base);
#pragma unroll
        for (int i = 0; i < kStepRows; ++i) {
            const int r = base + i * kStepGroups + group;
            if (r < a.d_k) {
                const float kk = k_s[r], qq = q_s[r];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[i][e] = keep * s[i][e] + kk * v[e];
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
        mine /= fmaxf(fabsf(nq), expf(-m)) + kMemoryFloor;
    }
    if (a.rows == nullptr) {
        if (owns) a.out[((size_t)t * a.heads + h) * a.d_v + col0 + c] = mine;
        return;
    }
    const float ss = block_sum(owns ? mine * mine : 0.f, scratch);
    if (owns) {
        const size_t at = (size_t)h * a.d_v + c;
        const float gate = gate_32(to_f32<T>(((const T*)a.gate)[(size_t)t * a.ld_gate + at]), a.gate_act);
        ((T*)a.rows)[(size_t)t * a.ld_rows + at] = from_f32<T>(mine * (1.f / sqrtf(ss / (float)a.d_v + a.eps)) * (a.weight ? a.weight[at] : 1.f) * gate);
    }
}

// ---------------------------------------------------------------------------------------------
// Many tokens: gates and running maximum, a CTA per (head, sequence).
constexpr int kGateWarps = 32;

template <typename T>
__global__ void __launch_bounds__(kGateWarps * 32)
memory_gates_kernel(MemoryArgs a) {
    __shared__ float run_a[kGateWarps], run_b[kGateWarps], run_m[kGateWarps], after;
    const int h = blockIdx.x, seq = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int first = a.cu_seqlens[seq], n = a.cu_seqlens[seq + 1] - first;
    pdl_launch_dependents();
    float* slot = a.state + (size_t)a.slots[seq] * a.slot_stride;
    float carry = *memory_m(a, slot, h, 0);
    const float b_i = a.bias_i[h], b_f = a.bias_f[h];
    pdl_wait();
    if (n <= 0) return;
    float* F = a.gates + (size_t)h * a.n_tokens + first;
    const size_t plane = (size_t)a.heads * a.n_tokens;
    if (threadIdx.x == 0) a.start_m[(size_t)seq * a.heads + h] = carry;
    for (int base = 0; base < n; base += kGateWarps * kRun) {
        const int t0 = base + warp * kRun + 2 * lane;
        float f[2] = {0.f, 0.f}, li[2] = {-INFINITY, -INFINITY};     // (tokens beyond the end change nothing)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            if (t0 + e < n) {
                const size_t t = (size_t)first + t0 + e;
                li[e] = log_input_gate(to_f32<T>(((const T*)a.zi)[t * a.ld_zi + h]) + b_i, a.cap);
                f[e] = log_forget_gate(to_f32<T>(((const T*)a.zf)[t * a.ld_zf + h]) + b_f, a.cap);
            }
        }
        float A = f[0] + f[1], B = fmaxf(li[0] + f[1], li[1]);
#pragma unroll
        for (int o = 1; o < 32; o *= 2) {
            const float pa = __shfl_up_sync(0xffffffffu, A, o), pb = __shfl_up_sync(0xffffffffu, B, o);
            if (lane >= o) {
                B = fmaxf(pb + A, B);
                A = pa + A;
            }
        }
        float xa = __shfl_up_sync(0xffffffffu, A, 1), xb = __shfl_up_sync(0xffffffffu, B, 1);
        if (lane == 0) { xa = 0.f; xb = -INFINITY; }
        if (lane == 31) { run_a[warp] = A; run_b[warp] = B; }
        __syncthreads();
        if (warp == 0) {      // the runs' own compositions, one per lane
            float ra = run_a[lane], rb = run_b[lane];
#pragma unroll
            for (int o = 1; o < 32; o *= 2) {
                const float pa = __shfl_up_sync(0xffffffffu, ra, o), pb = __shfl_up_sync(0xffffffffu, rb, o);
                if (lane >= o) {
                    rb = fmaxf(pb + ra, rb);
                    ra = pa + ra;
                }
            }
            const float ea = __shfl_up_sync(0xffffffffu, ra, 1), eb = __shfl_up_sync(0xffffffffu, rb, 1);
            run_m[lane] = lane == 0 ? carry : fmaxf(carry + ea, eb);
            if (lane == 31) after = fmaxf(carry + ra, rb);
        }
        __syncthreads();
        const float m0 = run_m[warp];
        float Fe[2] = {xa + f[0], 0.f}, be[2] = {fmaxf(xb + f[0], li[0]), 0.f};
        Fe[1] = Fe[0] + f[1];
        be[1] = fmaxf(be[0] + f[1], li[1]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            if (t0 + e < n) {
                F[t0 + e] = Fe[e];
                F[plane + t0 + e] = li[e];
                F[2 * plane + t0 + e] = fmaxf(m0 + Fe[e], be[e]);
                F[3 * plane + t0 + e] = f[e];
            }
        }
        carry = after;
        __syncthreads();       // (`after` and the runs' numbers may be written again)
    }
    // the maximum that goes with the memory the step leaves: the one written for its last token
    if (threadIdx.x < a.copies) *memory_m(a, slot, h, threadIdx.x) = F[2 * plane + n - 1];
}

// rows of q, k or v whose heads do not lie on the run kernels' grid, as rows whose heads are `pad` wide with zeros behind them
__global__ void __launch_bounds__(128)
memory_pad_kernel(const __nv_bfloat16* __restrict__ x, int ld_x, __nv_bfloat16* __restrict__ out, int heads, int d, int pad) {
    pdl_launch_dependents();
    pdl_wait();
    for (int u = threadIdx.x; u < heads * pad; u += 128) {
        const int h = u / pad, c = u % pad;
        out[(size_t)blockIdx.x * heads * pad + u] = c < d ? x[(size_t)blockIdx.x * ld_x + (size_t)h * d + c] : __float2bfloat16_rn(0.f);
    }
}

__device__ __forceinline__ size_t per_run(const MemoryArgs& a) { return ((size_t)a.d_k * a.d_v + a.d_k + 3) / 4 * 4; }
__device__ __forceinline__ float* run_at(const MemoryArgs& a, int seq, int run, int h) {
    return a.runs + ((size_t)(first_run(a.cu_seqlens, seq) + run) * a.heads + h) * per_run(a);
}
// m before run `run` of a sequence whose tokens start at row `seq0`
__device__ __forceinline__ float m_before(const MemoryArgs& a, int seq, int seq0, int run, int h) {
    return run == 0 ? a.start_m[(size_t)seq * a.heads + h]
                    : a.gates[((size_t)2 * a.heads + h) * a.n_tokens + seq0 + run * kRun - 1];
}

// (1) U[d_k, columns] = sum_j e^(F_n - F_j + i_j - m_n) k_j v_j^T of one run, and the same sum of the keys alone
template <int NS>
__global__ void __launch_bounds__(kRunThreads)
memory_run_sums_kernel(MemoryArgs a) {
    extern __shared__ __align__(16) uint8_t run_smem[];
    const int slices = (a.d_v + NS - 1) / NS;
    const int run = blockIdx.x / slices, col0 = (blockIdx.x % slices) * NS, h = blockIdx.y, seq = blockIdx.z;
    const int seq0 = a.cu_seqlens[seq], q_len = a.cu_seqlens[seq + 1] - seq0;
    pdl_launch_dependents();
    const int d_pad = (a.d_k + 15) / 16 * 16, ld = d_pad + 8, ldv = NS + 8;
    __nv_bfloat16* khi = reinterpret_cast<__nv_bfloat16*>(run_smem);
    __nv_bfloat16* klo = khi + kRun * ld;
    __nv_bfloat16* vs = klo + kRun * ld;
    __shared__ float w[kRun];
    const int first = seq0 + run * kRun, n = min(kRun, q_len - run * kRun);
    pdl_wait();
    if (n <= 0) return;
    load_tile(vs, ldv, a.vt + (size_t)first * a.ld_vt + (size_t)h * a.head_v + col0, a.ld_vt, n, NS, (a.d_v - col0 + 7) / 8 * 8);
    if (threadIdx.x < kRun) {
        const float* F = a.gates + (size_t)h * a.n_tokens + first;
        const size_t plane = (size_t)a.heads * a.n_tokens;
        const int j = threadIdx.x;
        w[j] = j < n ? expf((F[n - 1] - F[j]) + (F[plane + j] - F[2 * plane + n - 1])) : 0.f;
    }
    __syncthreads();
    const int per_row = d_pad / 8;
    for (int i = threadIdx.x; i < kRun * per_row; i += kRunThreads) {
        const int r = i / per_row, c = (i % per_row) * 8;
        uint32_t hi[4] = {0, 0, 0, 0}, lo[4] = {0, 0, 0, 0};
        if (r < n) {
            const float f = w[r];
            float x[8];
            load8(a.kt + (size_t)(first + r) * a.ld_kt + (size_t)h * a.head_qk + c, x);
#pragma unroll
            for (int e = 0; e < 4; ++e) split_pair(x[2 * e] * f, x[2 * e + 1] * f, hi[e], lo[e]);
        }
        *reinterpret_cast<uint4*>(khi + (size_t)r * ld + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(klo + (size_t)r * ld + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    copies_done();
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, mi = lane >> 3, mr = lane & 7, gq = lane >> 2, tq = lane & 3;
    float* U = run_at(a, seq, run, h);
    if (col0 == 0) {
        for (int i = threadIdx.x; i < a.d_k; i += kRunThreads) {
            float sum = 0.f;
            for (int r = 0; r < n; ++r) sum += __bfloat162float(khi[(size_t)r * ld + i]) + __bfloat162float(klo[(size_t)r * ld + i]);
            U[(size_t)a.d_k * a.d_v + i] = sum;
        }
    }
    for (int m = warp; m < d_pad / 16; m += kRunThreads / 32) {
        float acc[NS / 8][4];
#pragma unroll
        for (int j = 0; j < NS / 8; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
#pragma unroll
        for (int kk = 0; kk < kRun / 16; ++kk) {
            if (kk * 16 >= n) break;
            uint32_t ah[4], al[4];      // the weighted keys transposed
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

// (2) per element of S and n, run after run: the run's sum is replaced by the memory before the run (S as its hi and lo part);
// the memory after the last run goes back to the slot.  Sixteen runs' sums are asked for at once.
__global__ void __launch_bounds__(256)
memory_carry_kernel(MemoryArgs a) {
    __shared__ float keep[16];
    const int h = blockIdx.y, seq = blockIdx.z;
    const int n_s = a.d_k * a.d_v, e = blockIdx.x * 256 + threadIdx.x;
    const int seq0 = a.cu_seqlens[seq], q_len = a.cu_seqlens[seq + 1] - seq0;
    const int n_runs = (q_len + kRun - 1) / kRun;
    pdl_launch_dependents();
    pdl_wait();
    if (n_runs == 0) return;
    const bool live = e < n_s + a.d_k, is_n = e >= n_s;
    float* slot = a.state + (size_t)a.slots[seq] * a.slot_stride;
    float* S = is_n ? memory_n(a, slot, h, 0) + (e - n_s) : slot + (size_t)h * n_s + e;
    float carry = live ? *S : 0.f;
    const float* F = a.gates + (size_t)h * a.n_tokens + seq0;
    const float* M = F + (size_t)2 * a.heads * a.n_tokens;
    const size_t step = (size_t)a.heads * per_run(a);
    float* u = run_at(a, seq, 0, h) + e;
    for (int r0 = 0; r0 < n_runs; r0 += 16) {
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) x[i] = live && r0 + i < n_runs ? u[(size_t)(r0 + i) * step] : 0.f;
        __syncthreads();
        if (threadIdx.x < 16 && r0 + (int)threadIdx.x < n_runs) {
            const int run = r0 + threadIdx.x, last = min(q_len, (run + 1) * kRun) - 1;
            keep[threadIdx.x] = expf(F[last] + (m_before(a, seq, seq0, run, h) - M[last]));
        }
        __syncthreads();
        if (!live) continue;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            if (r0 + i < n_runs) {
                if (is_n) {
                    u[(size_t)(r0 + i) * step] = carry;
                } else {
                    const __nv_bfloat16 hi = __float2bfloat16_rn(carry);
                    const __nv_bfloat162 both = __halves2bfloat162(hi, __float2bfloat16_rn(carry - __bfloat162float(hi)));
                    u[(size_t)(r0 + i) * step] = __uint_as_float(*reinterpret_cast<const uint32_t*>(&both));
                }
                carry = keep[i] * carry + x[i];
            }
        }
    }
    if (!live) return;
    if (is_n) {
        for (int c = 0; c < a.copies; ++c) memory_n(a, slot, h, c)[e - n_s] = carry;
    } else {
        *S = carry;
    }
}

// (3) outputs of one run
template <int NS>
__global__ void __launch_bounds__(kRunThreads)
memory_outputs_kernel(MemoryArgs a) {
    extern __shared__ __align__(16) uint8_t run_smem[];
    const int slices = (a.d_v + NS - 1) / NS;
    const int run = blockIdx.x / slices, col0 = (blockIdx.x % slices) * NS, h = blockIdx.y, seq = blockIdx.z;
    const int seq0 = a.cu_seqlens[seq], q_len = a.cu_seqlens[seq + 1] - seq0;
    pdl_launch_dependents();
    const int d_pad = (a.d_k + 15) / 16 * 16, ld = d_pad + 8, ldv = NS + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(run_smem);
    __nv_bfloat16* ks = qs + kRun * ld;
    __nv_bfloat16* vs = ks + kRun * ld;
    __nv_bfloat16* shi = vs + kRun * ldv;
    __nv_bfloat16* slo = shi + d_pad * ldv;
    float* n_s = reinterpret_cast<float*>(slo + d_pad * ldv);      // [d_pad]
    // weights e^(w_i + w_j), e^w_before of the memory before the run, and what the divisor is at least
    __shared__ float w_i[kRun], w_j[kRun], before[kRun], least[kRun];
    const int first = seq0 + run * kRun, n = min(kRun, q_len - run * kRun);
    pdl_wait();
    if (n <= 0) return;
    load_tile(qs, ld, a.qt + (size_t)first * a.ld_qt + (size_t)h * a.head_qk, a.ld_qt, n, d_pad, d_pad);
    load_tile(ks, ld, a.kt + (size_t)first * a.ld_kt + (size_t)h * a.head_qk, a.ld_kt, n, d_pad, d_pad);
    load_tile(vs, ldv, a.vt + (size_t)first * a.ld_vt + (size_t)h * a.head_v + col0, a.ld_vt, n, NS, (a.d_v - col0 + 7) / 8 * 8);
    const float* U = run_at(a, seq, run, h);
    const float* F = a.gates + (size_t)h * a.n_tokens + first;
    const size_t plane = (size_t)a.heads * a.n_tokens;
    const int mine = min((int)threadIdx.x % kRun, n - 1);      // (asked for before the memory's tiles, used behind them)
    const float f = F[mine], log_in = F[plane + mine], m = F[2 * plane + mine], m_first = m_before(a, seq, seq0, run, h);
    load_state_parts<NS>(shi, slo, ldv, reinterpret_cast<const uint32_t*>(U), a.d_k, a.d_v, col0, d_pad);
    for (int i = threadIdx.x; i < d_pad; i += kRunThreads) n_s[i] = i < a.d_k ? U[(size_t)a.d_k * a.d_v + i] : 0.f;
    if (threadIdx.x < kRun) {
        w_i[threadIdx.x] = f - m;
        w_j[threadIdx.x] = log_in - f;
        before[threadIdx.x] = expf(f + (m_first - m));
        least[threadIdx.x] = expf(-m);
    }
    copies_done();
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
    // scores against the run's tokens up to this warp's last row, and the read-out of the memory before the run
    for (int kk = 0; kk < d_pad / 16; ++kk) {
        uint32_t ah[4];
        ldsm4(ah, qs + (row0 + (mi & 1) * 8 + mr) * ld + kk * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int j = 0; j < kRun / 16; ++j) {
            if (j <= warp) {
                uint32_t bh[4];
                ldsm4(bh, ks + (j * 16 + (mi >> 1) * 8 + mr) * ld + kk * 16 + (mi & 1) * 8);
                mma_run(sc[2 * j], ah, bh[0], bh[1]);
                mma_run(sc[2 * j + 1], ah, bh[2], bh[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < NS / 16; ++j) {
            uint32_t bh[4], bl[4];
            const int bt = (kk * 16 + (mi & 1) * 8 + mr) * ldv + j * 16 + (mi >> 1) * 8;
            ldsm4t(bh, shi + bt);
            ldsm4t(bl, slo + bt);
            mma_run(o[2 * j], ah, bh[0], bh[1]);
            mma_run(o[2 * j + 1], ah, bh[2], bh[3]);
            mma_run(o[2 * j], ah, bl[0], bl[1]);
            mma_run(o[2 * j + 1], ah, bl[2], bl[3]);
        }
    }
    const int i0 = row0 + gq, i1 = i0 + 8;
    const float f0 = before[i0], f1 = before[i1];
    // n . q of the memory before the run: the four lanes of a row share its numbers
    float nq[2] = {0.f, 0.f};
    for (int c = 2 * tq; c < d_pad; c += 8) {
        const float2 nn = *reinterpret_cast<const float2*>(n_s + c);
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
            const uint32_t q2 = *reinterpret_cast<const uint32_t*>(qs + (size_t)(hh ? i1 : i0) * ld + c);
            nq[hh] += nn.x * __uint_as_float(q2 << 16) + nn.y * __uint_as_float(q2 & 0xffff0000u);
        }
    }
    nq[0] *= f0;
    nq[1] *= f1;
#pragma unroll
    for (int j = 0; j < NS / 8; ++j) {
        o[j][0] *= f0; o[j][1] *= f0;
        o[j][2] *= f1; o[j][3] *= f1;
    }
    // the weighted scores times the run's values
    const float wi0 = w_i[i0], wi1 = w_i[i1];
#pragma unroll
    for (int j = 0; j < kRun / 16; ++j) {
        if (j > warp) continue;
        uint32_t ah[4], al[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int c = j * 16 + half * 8 + 2 * tq;
            const float wa = w_j[c], wb = w_j[c + 1];
            float p[4];
            p[0] = c <= i0 ? sc[2 * j + half][0] * expf(wi0 + wa) : 0.f;
            p[1] = c + 1 <= i0 ? sc[2 * j + half][1] * expf(wi0 + wb) : 0.f;
            p[2] = c <= i1 ? sc[2 * j + half][2] * expf(wi1 + wa) : 0.f;
            p[3] = c + 1 <= i1 ? sc[2 * j + half][3] * expf(wi1 + wb) : 0.f;
            nq[0] += p[0] + p[1];
            nq[1] += p[2] + p[3];
#pragma unroll
            for (int r = 0; r < 2; ++r) split_pair(p[2 * r], p[2 * r + 1], ah[2 * half + r], al[2 * half + r]);
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
        nq[hh] += __shfl_xor_sync(0xffffffffu, nq[hh], 1);
        nq[hh] += __shfl_xor_sync(0xffffffffu, nq[hh], 2);
        const int i = hh ? i1 : i0;
        const float mul = a.q_scale / (fmaxf(fabsf(nq[hh] * a.q_scale), least[i]) + kMemoryFloor);
#pragma unroll
        for (int j = 0; j < NS / 8; ++j) { o[j][2 * hh] *= mul; o[j][2 * hh + 1] *= mul; }
        if (a.rows != nullptr) {
            // the head is finished here: its numbers lie in the four lanes of the row (columns beyond d_v are zero)
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < NS / 8; ++j) ss += o[j][2 * hh] * o[j][2 * hh] + o[j][2 * hh + 1] * o[j][2 * hh + 1];
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            if (i >= n) continue;
            const float scale = 1.f / sqrtf(ss / (float)a.d_v + a.eps);
            const size_t t = (size_t)first + i;
            const __nv_bfloat16* gate = (const __nv_bfloat16*)a.gate + t * a.ld_gate + (size_t)h * a.d_v;
            __nv_bfloat16* dst = (__nv_bfloat16*)a.rows + t * a.ld_rows + (size_t)h * a.d_v;
            const float* wt = a.weight ? a.weight + (size_t)h * a.d_v : nullptr;
            const bool pairs = (((uintptr_t)gate | (uintptr_t)dst) & 3) == 0;
            uint32_t g2[NS / 8];      // (all asked for before the first result is stored)
#pragma unroll
            for (int j = 0; j < NS / 8; ++j)
                g2[j] = pairs && j * 8 + 2 * tq + 1 < a.d_v ? __ldg(reinterpret_cast<const uint32_t*>(gate + j * 8 + 2 * tq)) : 0u;
#pragma unroll
            for (int j = 0; j < NS / 8; ++j) {
                const int c = j * 8 + 2 * tq;
                if (c + 1 < a.d_v && pairs) {
                    *reinterpret_cast<uint32_t*>(dst + c) =
                        pack_pair(o[j][2 * hh] * scale * (wt ? __ldg(wt + c) : 1.f) * gate_16(__uint_as_float(g2[j] << 16), a.gate_act),
                                  o[j][2 * hh + 1] * scale * (wt ? __ldg(wt + c + 1) : 1.f) * gate_16(__uint_as_float(g2[j] & 0xffff0000u), a.gate_act));
                } else {
                    for (int e = 0; e < 2; ++e)
                        if (c + e < a.d_v)
                            dst[c + e] = __float2bfloat16_rn(o[j][2 * hh + e] * scale * (wt ? wt[c + e] : 1.f) * gate_16(__bfloat162float(gate[c + e]), a.gate_act));
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

// What the scan leaves per token and head, the d_v read-outs and n . q behind them, as quotients; and the scan's last n, which
// it wrote into the first copy, into the others (blocks of the second grid row).
__global__ void __launch_bounds__(128)
memory_divide_kernel(MemoryArgs a, const float* __restrict__ scanned) {
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (blockIdx.y == 1) {
        if (row >= a.n_seqs * a.heads) return;
        const int seq = row / a.heads, h = row % a.heads;
        if (a.cu_seqlens[seq + 1] == a.cu_seqlens[seq]) return;
        float* slot = a.state + (size_t)a.slots[seq] * a.slot_stride;
        for (int c = 1; c < a.copies; ++c)
            for (int i = lane; i < a.d_k; i += 32) memory_n(a, slot, h, c)[i] = memory_n(a, slot, h, 0)[i];
        return;
    }
    if (row >= a.n_tokens * a.heads) return;
    const int t = row / a.heads, h = row % a.heads;
    const float* x = scanned + (size_t)row * (a.d_v + 1);
    const float m = a.gates[((size_t)2 * a.heads + h) * a.n_tokens + t];
    const float total = fmaxf(fabsf(x[a.d_v]), expf(-m)) + kMemoryFloor;
    for (int c = lane; c < a.d_v; c += 32) a.out[(size_t)row * a.d_v + c] = x[c] / total;
}

static size_t outputs_smem(int d_k, int ns) {
    const int d_pad = (d_k + 15) / 16 * 16;
    return sizeof(__nv_bfloat16) * ((size_t)2 * kRun * (d_pad + 8) + (size_t)kRun * (ns + 8) + (size_t)2 * d_pad * (ns + 8)) + sizeof(float) * d_pad;
}
static size_t sums_smem(int d_k, int ns) {
    const int d_pad = (d_k + 15) / 16 * 16;
    return sizeof(__nv_bfloat16) * ((size_t)2 * kRun * (d_pad + 8) + (size_t)kRun * (ns + 8));
}
constexpr size_t kMostSmem = 227 * 1024 - 2048;    // (two kilobytes for the static part)

// columns of the values a CTA takes: all of a head's up to 128 where shared memory allows, else slices of 64; 0: no fit
static int run_columns(int d_k, int d_v) {
    if (d_v > 64 && outputs_smem(d_k, 128) <= kMostSmem) return 128;
    return outputs_smem(d_k, 64) <= kMostSmem ? 64 : 0;
}
static size_t run_floats(int n_tokens, int n_seqs, int heads, int d_k, int d_v) {
    return (size_t)(n_tokens / kRun + n_seqs + 1) * heads * (((size_t)d_k * d_v + d_k + 3) / 4 * 4);
}
static size_t gate_floats(int n_tokens, int n_seqs, int heads) {
    return ((size_t)4 * heads * n_tokens + (size_t)n_seqs * heads + 3) / 4 * 4;
}

template <int NS>
static int launch_runs(const MemoryArgs& a, int max_q_len, cudaStream_t stream) {
    const size_t s1 = sums_smem(a.d_k, NS), s3 = outputs_smem(a.d_k, NS);
    static size_t have1 = 48 * 1024, have3 = 48 * 1024;
    if (s1 > have1) {
        const int e = (int)cudaFuncSetAttribute(memory_run_sums_kernel<NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        if (e != 0) return e;
        have1 = s1;
    }
    if (s3 > have3) {
        const int e = (int)cudaFuncSetAttribute(memory_outputs_kernel<NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
        if (e != 0) return e;
        have3 = s3;
    }
    const int n_runs = (max_q_len + kRun - 1) / kRun, slices = (a.d_v + NS - 1) / NS;
    const dim3 grid(n_runs * slices, a.heads, a.n_seqs);
    int st = launch_pdl(memory_run_sums_kernel<NS>, grid, dim3(kRunThreads), s1, stream, a);
    if (st != 0) return st;
    st = launch_pdl(memory_carry_kernel, dim3((a.d_k * (a.d_v + 1) + 255) / 256, a.heads, a.n_seqs), dim3(256), 0, stream, a);
    if (st != 0) return st;
    return launch_pdl(memory_outputs_kernel<NS>, grid, dim3(kRunThreads), s3, stream, a);
}

template <typename T, int VEC, int TPR>
static int launch_memory_step(const MemoryArgs& a, cudaStream_t stream) {
    constexpr int COLS = VEC * TPR;
    const size_t smem = sizeof(float) * ((size_t)2 * a.d_k + (size_t)kStepGroups * COLS);
    const dim3 grid((a.d_v + COLS - 1) / COLS, a.heads, a.n_seqs);
    return launch_pdl(memory_step_kernel<T, VEC, TPR>, grid, dim3(kStepGroups * TPR), smem, stream, a);
}

static int step_columns(int d_v) { return d_v % 4 != 0 ? 32 : d_v <= 64 ? 64 : 128; }

}  // namespace b200

// How many copies of n and m a head keeps: the slices of its columns that the one-token kernel takes.
extern "C" int b200_matrix_memory_copies(int d_v) { return (d_v + b200::step_columns(d_v) - 1) / b200::step_columns(d_v); }
// Columns of a head's values that one CTA of the run kernels takes (0: they do not take this key size).
extern "C" int b200_matrix_memory_columns(int d_k, int d_v) { return b200::run_columns(d_k, d_v); }
// Floats of scratch for the gates (steps of more than one token per sequence), and for those and the run kernels.
extern "C" long long b200_matrix_memory_gate_floats(int n_tokens, int n_seqs, int heads) { return (long long)b200::gate_floats(n_tokens, n_seqs, heads); }
extern "C" long long b200_matrix_memory_scratch(int n_tokens, int n_seqs, int heads, int d_k, int d_v) {
    const long long d_pad = (d_k + 15) / 16 * 16, v_pad = (d_v + 7) / 8 * 8;
    return (long long)(b200::gate_floats(n_tokens, n_seqs, heads) + b200::run_floats(n_tokens, n_seqs, heads, d_k, d_v)) +
           ((2 * d_pad + v_pad) * n_tokens * heads + 1) / 2;
}

// stage 0: the whole recurrence (one token per sequence, or the run kernels over bfloat16 operands); 1: gates alone, for the
// scan; 2: the quotients of what the scan left in `scanned` [T, heads, d_v + 1].  `scratch` as the functions above say.
// out: float32 [T, heads d_v], or rows (not null): the finished heads into [T, ld_rows].
extern "C" int b200_matrix_memory(int stage, const void* q, int ld_q, const void* k, int ld_k, const void* v, int ld_v, const void* zi,
                                  int ld_zi, const void* zf, int ld_zf, const float* bias_i, const float* bias_f, float cap,
                                  float* state, long long slot_stride, int copies, const int* slots, const int* cu_seqlens, float* out,
                                  float* scratch, const float* scanned, int dtype, int n_tokens, int n_seqs, int max_q_len, int heads,
                                  int d_k, int d_v, float q_scale, const float* weight, const void* gate, int ld_gate, int gate_act,
                                  void* rows, int ld_rows, float eps, cudaStream_t stream) {
    using namespace b200;
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (heads < 1 || heads > 65535 || n_seqs > 65535 || d_k < 1 || d_v < 1 || d_k > kStepMostKeys || !(cap > 0.f)) return kErrBadArgument;
    if (copies != b200_matrix_memory_copies(d_v) || copies > 1024) return kErrBadArgument;
    if (rows != nullptr && (out != nullptr || !gate || ld_rows < heads * d_v || ld_gate < heads * d_v)) return kErrBadArgument;
    MemoryArgs a = {};
    a.q = q; a.k = k; a.v = v; a.ld_q = ld_q; a.ld_k = ld_k; a.ld_v = ld_v;
    a.zi = zi; a.zf = zf; a.ld_zi = ld_zi; a.ld_zf = ld_zf; a.bias_i = bias_i; a.bias_f = bias_f; a.cap = cap;
    a.state = state; a.slot_stride = (size_t)slot_stride; a.copies = copies; a.slots = slots; a.cu_seqlens = cu_seqlens; a.out = out;
    a.n_tokens = n_tokens; a.n_seqs = n_seqs; a.heads = heads; a.d_k = d_k; a.d_v = d_v; a.q_scale = q_scale;
    a.weight = weight; a.gate = gate; a.ld_gate = ld_gate; a.gate_act = gate_act; a.rows = rows; a.ld_rows = ld_rows; a.eps = eps;
    a.gates = scratch;
    a.start_m = scratch + (size_t)4 * heads * n_tokens;
    if (stage == 0 && n_tokens == n_seqs) {
        if (out == nullptr && (rows == nullptr || copies > 1)) return kErrBadArgument;
        const bool vec = d_v % 4 == 0;
        if (vec && (slot_stride % 4 != 0 || ((uintptr_t)state & 15))) return kErrBadArgument;
        B200_DISPATCH_DTYPE(dtype, T,
            if (!vec) return launch_memory_step<T, 1, 32>(a, stream);
            if (d_v <= 64) return launch_memory_step<T, 4, 16>(a, stream);
            return launch_memory_step<T, 4, 32>(a, stream));
        return 0;
    }
    if (!scratch || ((uintptr_t)scratch & 15)) return kErrBadArgument;
    if (stage == 2) {
        if (out == nullptr || scanned == nullptr) return kErrBadArgument;
        const long long most = (long long)(n_tokens > n_seqs ? n_tokens : n_seqs) * heads;
        memory_divide_kernel<<<dim3((unsigned)((most + 3) / 4), copies > 1 ? 2 : 1), 128, 0, stream>>>(a, scanned);
        return launch_status();
    }
    if (stage != 0 && stage != 1) return kErrBadArgument;
    const int ns = run_columns(d_k, d_v);
    if (stage == 0) {
        if (dtype != kBF16 || ns == 0) return kErrUnsupportedSize;
        if (out == nullptr && (rows == nullptr || d_v > ns)) return kErrBadArgument;
    }
    B200_DISPATCH_DTYPE(dtype, T,
        const int st = launch_pdl(memory_gates_kernel<T>, dim3(heads, n_seqs), dim3(kGateWarps * 32), 0, stream, a);
        if (st != 0 || stage == 1) return st);
    a.runs = scratch + gate_floats(n_tokens, n_seqs, heads);
    __nv_bfloat16* room = reinterpret_cast<__nv_bfloat16*>(a.runs + run_floats(n_tokens, n_seqs, heads, d_k, d_v));
    const int d_pad = (d_k + 15) / 16 * 16, v_pad = (d_v + 7) / 8 * 8;
    auto ready = [](const void* x, int ld, int d, int grid) { return d % grid == 0 && ld % 8 == 0 && ((uintptr_t)x & 15) == 0; };
    int st = 0;
    auto padded = [&](const void* x, int ld, int d, int pad) {
        __nv_bfloat16* at = room;
        room += (size_t)n_tokens * heads * pad;
        if (st == 0) st = launch_pdl(memory_pad_kernel, dim3(n_tokens), dim3(128), 0, stream, (const __nv_bfloat16*)x, ld, at, heads, d, pad);
        return (const __nv_bfloat16*)at;
    };
    a.qt = (const __nv_bfloat16*)q; a.kt = (const __nv_bfloat16*)k; a.vt = (const __nv_bfloat16*)v;
    a.ld_qt = ld_q; a.ld_kt = ld_k; a.ld_vt = ld_v; a.head_qk = d_k; a.head_v = d_v;
    if (!ready(q, ld_q, d_k, 16) || !ready(k, ld_k, d_k, 16)) {
        a.qt = padded(q, ld_q, d_k, d_pad);
        a.kt = padded(k, ld_k, d_k, d_pad);
        a.ld_qt = a.ld_kt = heads * d_pad;
        a.head_qk = d_pad;
    }
    if (!ready(v, ld_v, d_v, 8)) {
        a.vt = padded(v, ld_v, d_v, v_pad);
        a.ld_vt = heads * v_pad;
        a.head_v = v_pad;
    }
    if (st != 0) return st;
    return ns == 128 ? launch_runs<128>(a, max_q_len, stream) : launch_runs<64>(a, max_q_len, stream);
}
