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
// tensor-core operand has 16: turned queries and keys, the decayed keys, the decayed scores and the state therefore enter as
// the sum of two bfloat16 numbers (x = hi + lo, 16 bits of mantissa), products of two such sums without the lo lo term; sums
// are 32-bit.  The powers of g are exact to 32-bit rounding (powf).  Projections, with SiLU or without, enter as the one
// bfloat16 number they are stored as.  A sequence's runs start at the step's first token of the sequence; the last one may be
// short.  The tiles are read as they lie in memory, 16 bytes at a time: where queries and keys have to be turned or
// activated, or a head's size is off that grid, a kernel in front of the three leaves them so (fixed_decay_prepare).
#include "run_tiles.cuh"

namespace b200 {

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
    float* out;             // [T, heads d_v] 32-bit, or null when the head is finished here
    float* runs;            // scratch of the prompt kernels: [run][head][d_k][d_v]; behind the second one the state before the
                            // run as (hi, lo) pairs of bfloat16 in the place of each number
    // how the prompt kernels read the operands: rows of bfloat16 on 16-byte boundaries, head h at column h * head_qk (head_v)
    const __nv_bfloat16* qt[2];   // hi and lo (the second where the operand has two parts)
    const __nv_bfloat16* kt[2];
    const __nv_bfloat16* vt;
    int ld_qt, ld_kt, ld_vt, head_qk, head_v;
    int n_tokens, heads, d_k, d_v, pairs, qk_silu, v_silu;
    float q_scale;
    // the finished head: o / sqrt(mean(o^2) + eps) * act(gate) * mul into columns of a buffer of the operands' type
    const void* gate;       // [T, ld_gate], head h at column h d_v
    int ld_gate, gate_act;  // 0 sigmoid, 1 SiLU
    void* rows;             // [T, ld_rows]
    int ld_rows;
    float eps, mul;
};

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

// Queries, keys and values as the run kernels read them, a CTA per token: heads d_pad (v_pad) wide with zeros behind them,
// activated and turned, q and k in `parts` bfloat16 numbers each.  Angles once per token.
struct PrepareRows {
    __nv_bfloat16* qk[2][2];    // [q or k][hi or lo], rows of heads * d_pad; null: left as they are
    __nv_bfloat16* v;           // rows of heads * v_pad, or null
    int d_pad, v_pad;
};

__global__ void __launch_bounds__(128)
fixed_decay_prepare_kernel(FixedDecayArgs a, PrepareRows p) {
    extern __shared__ float turn[];      // [pairs] cos, [pairs] sin
    const int t = blockIdx.x;
    pdl_launch_dependents();
    if (a.pairs > 0) {
        const float pos = (float)a.positions[t];
        for (int i = threadIdx.x; i < a.pairs; i += 128) sincosf(pos * a.inv_freq[i], &turn[a.pairs + i], &turn[i]);
        __syncthreads();
    }
    pdl_wait();
    if (p.qk[0][0] != nullptr) {
        const bool vec = a.d_k % 4 == 0 && a.pairs % 4 == 0 && a.ld_q % 4 == 0 && a.ld_k % 4 == 0 && (((uintptr_t)a.q | (uintptr_t)a.k) & 7) == 0;
        const int chunks = p.d_pad / 4, units = 2 * a.heads * chunks;      // four neighbouring numbers of a head
        for (int u = threadIdx.x; u < units; u += 128) {
            const int which = u / (a.heads * chunks), h = (u / chunks) % a.heads, c = (u % chunks) * 4;
            const __nv_bfloat16* x = (which ? (const __nv_bfloat16*)a.k + (size_t)t * a.ld_k : (const __nv_bfloat16*)a.q + (size_t)t * a.ld_q) +
                                     (size_t)h * a.d_k;
            float y[4];
            if (vec) {      // (the four numbers, and their partners, lie side by side)
                const bool first = c < a.pairs, turned = c < 2 * a.pairs;
                const int o = !turned ? c : first ? c + a.pairs : c - a.pairs, f = first ? c : o;
                float z[4] = {0.f, 0.f, 0.f, 0.f}, zo[4] = {0.f, 0.f, 0.f, 0.f};
                if (c < a.d_k) {
                    load4(x + c, z);
                    if (turned) load4(x + o, zo);
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    if (a.qk_silu) { z[e] = silu_32(z[e]); zo[e] = silu_32(zo[e]); }
                    y[e] = !turned ? z[e] : z[e] * turn[f + e] + (first ? -zo[e] : zo[e]) * turn[a.pairs + f + e];
                }
            } else
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = c + e;
                float z = i < a.d_k ? __bfloat162float(x[i]) : 0.f;
                if (a.qk_silu) z = silu_32(z);
                if (i < 2 * a.pairs) {
                    const bool first = i < a.pairs;
                    const int o = first ? i + a.pairs : i - a.pairs, f = first ? i : o;
                    float zo = __bfloat162float(x[o]);
                    if (a.qk_silu) zo = silu_32(zo);
                    z = first ? z * turn[f] - zo * turn[a.pairs + f] : z * turn[f] + zo * turn[a.pairs + f];
                }
                y[e] = z;
            }
            const size_t at = ((size_t)t * a.heads + h) * p.d_pad + c;
            uint32_t hi[2], lo[2];
            split_pair(y[0], y[1], hi[0], lo[0]);
            split_pair(y[2], y[3], hi[1], lo[1]);
            *reinterpret_cast<uint2*>(p.qk[which][0] + at) = make_uint2(hi[0], hi[1]);
            if (p.qk[which][1] != nullptr) *reinterpret_cast<uint2*>(p.qk[which][1] + at) = make_uint2(lo[0], lo[1]);
        }
    }
    if (p.v != nullptr) {
        const __nv_bfloat16* x = (const __nv_bfloat16*)a.v + (size_t)t * a.ld_v;
        for (int u = threadIdx.x; u < a.heads * p.v_pad; u += 128) {
            const int h = u / p.v_pad, c = u % p.v_pad;
            const float z = c < a.d_v ? __bfloat162float(x[(size_t)h * a.d_v + c]) : 0.f;
            p.v[(size_t)t * a.heads * p.v_pad + u] = __float2bfloat16_rn(a.v_silu ? silu_32(z) : z);
        }
    }
}

// powers g^0 .. g^kRun in shared memory
__device__ __forceinline__ void powers(float* pw, float g) {
    for (int i = threadIdx.x; i <= kRun; i += kRunThreads) pw[i] = i == 0 ? 1.f : powf(g, (float)i);
}

// (1) U[d_k, columns] = sum_j g^(n - 1 - j) k_j v_j^T of one run
template <int NS, int PARTS>
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
    __shared__ float pw[kRun + 1];
    powers(pw, a.decay[h]);
    const int first = seq0 + run * kRun, n = min(kRun, q_len - run * kRun);
    __syncthreads();
    pdl_wait();
    if (n <= 0) return;
    load_tile(vs, ldv, a.vt + (size_t)first * a.ld_vt + (size_t)h * a.head_v + col0, a.ld_vt, n, NS, (a.d_v - col0 + 7) / 8 * 8);
    // the keys times the decay until the run's end, in two parts again
    const int per_row = d_pad / 8;
    for (int i = threadIdx.x; i < kRun * per_row; i += kRunThreads) {
        const int r = i / per_row, c = (i % per_row) * 8;
        uint32_t hi[4] = {0, 0, 0, 0}, lo[4] = {0, 0, 0, 0};
        if (r < n) {
            const float f = pw[n - 1 - r];
            const size_t at = (size_t)(first + r) * a.ld_kt + (size_t)h * a.head_qk + c;
            float x[8];
            load8(a.kt[0] + at, x);
            if constexpr (PARTS == 2) {
                float y[8];
                load8(a.kt[1] + at, y);
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] += y[e];
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) split_pair(x[2 * e] * f, x[2 * e + 1] * f, hi[e], lo[e]);
        }
        *reinterpret_cast<uint4*>(khi + (size_t)r * ld + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(klo + (size_t)r * ld + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    copies_done();
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

// (2) per element, run after run: the scratch's run sum is replaced by the state before the run, as its hi and lo part; the
// state after the last run goes back to the slot.  Sixteen runs' sums are asked for at once.
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
    for (int r0 = 0; r0 < n_runs; r0 += 16) {
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) x[i] = r0 + i < n_runs ? u[(size_t)(r0 + i) * step] : 0.f;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            if (r0 + i < n_runs) {
                const __nv_bfloat16 hi = __float2bfloat16_rn(carry);
                const __nv_bfloat162 both = __halves2bfloat162(hi, __float2bfloat16_rn(carry - __bfloat162float(hi)));
                u[(size_t)(r0 + i) * step] = __uint_as_float(*reinterpret_cast<const uint32_t*>(&both));
                carry = (r0 + i == n_runs - 1 ? g_last : g_run) * carry + x[i];
            }
        }
    }
    *S = carry;
}

// (3) outputs of one run
template <int NS, int PARTS>
__global__ void __launch_bounds__(kRunThreads)
fixed_decay_outputs_kernel(FixedDecayArgs a) {
    extern __shared__ __align__(16) uint8_t run_smem[];
    const int slices = (a.d_v + NS - 1) / NS;
    const int run = blockIdx.x / slices, col0 = (blockIdx.x % slices) * NS, h = blockIdx.y, seq = blockIdx.z;
    const int seq0 = a.cu_seqlens[seq], q_len = a.cu_seqlens[seq + 1] - seq0;
    pdl_launch_dependents();
    const int d_pad = (a.d_k + 15) / 16 * 16, ld = d_pad + 8, ldv = NS + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(run_smem);      // PARTS tiles
    __nv_bfloat16* ks = qs + PARTS * kRun * ld;
    __nv_bfloat16* vs = ks + PARTS * kRun * ld;
    __nv_bfloat16* shi = vs + kRun * ldv;
    __nv_bfloat16* slo = shi + d_pad * ldv;
    __shared__ float pw[kRun + 1];
    powers(pw, a.decay[h]);
    const int first = seq0 + run * kRun, n = min(kRun, q_len - run * kRun);
    pdl_wait();
    if (n <= 0) return;
#pragma unroll
    for (int p = 0; p < PARTS; ++p) {
        load_tile(qs + p * kRun * ld, ld, a.qt[p] + (size_t)first * a.ld_qt + (size_t)h * a.head_qk, a.ld_qt, n, d_pad, d_pad);
        load_tile(ks + p * kRun * ld, ld, a.kt[p] + (size_t)first * a.ld_kt + (size_t)h * a.head_qk, a.ld_kt, n, d_pad, d_pad);
    }
    load_tile(vs, ldv, a.vt + (size_t)first * a.ld_vt + (size_t)h * a.head_v + col0, a.ld_vt, n, NS, (a.d_v - col0 + 7) / 8 * 8);
    load_state_parts<NS>(shi, slo, ldv, reinterpret_cast<const uint32_t*>(a.runs) + ((size_t)(first_run(a.cu_seqlens, seq) + run) * a.heads + h) * a.d_k * a.d_v, a.d_k, a.d_v, col0, d_pad);
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
    // scores against the run's tokens up to this warp's last row, and the read-out of the state before the run
    for (int kk = 0; kk < d_pad / 16; ++kk) {
        uint32_t ah[4], al[4];
        const int at = (row0 + (mi & 1) * 8 + mr) * ld + kk * 16 + (mi >> 1) * 8;
        ldsm4(ah, qs + at);
        if constexpr (PARTS == 2) ldsm4(al, qs + kRun * ld + at);
#pragma unroll
        for (int j = 0; j < kRun / 16; ++j) {
            if (j <= warp) {
                uint32_t bh[4], bl[4];
                const int bt = (j * 16 + (mi >> 1) * 8 + mr) * ld + kk * 16 + (mi & 1) * 8;
                ldsm4(bh, ks + bt);
                mma_run(sc[2 * j], ah, bh[0], bh[1]);
                mma_run(sc[2 * j + 1], ah, bh[2], bh[3]);
                if constexpr (PARTS == 2) {
                    ldsm4(bl, ks + kRun * ld + bt);
                    mma_run(sc[2 * j], ah, bl[0], bl[1]);
                    mma_run(sc[2 * j + 1], ah, bl[2], bl[3]);
                    mma_run(sc[2 * j], al, bh[0], bh[1]);
                    mma_run(sc[2 * j + 1], al, bh[2], bh[3]);
                }
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
            if constexpr (PARTS == 2) {
                mma_run(o[2 * j], al, bh[0], bh[1]);
                mma_run(o[2 * j + 1], al, bh[2], bh[3]);
            }
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
    for (int j = 0; j < NS / 8; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[j][i] *= a.q_scale;
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
            uint32_t g2[NS / 8];      // (all asked for before the first result is stored)
#pragma unroll
            for (int j = 0; j < NS / 8; ++j)
                g2[j] = pairs && j * 8 + 2 * tq + 1 < a.d_v ? __ldg(reinterpret_cast<const uint32_t*>(gate + j * 8 + 2 * tq)) : 0u;
#pragma unroll
            for (int j = 0; j < NS / 8; ++j) {
                const int c = j * 8 + 2 * tq;
                if (c + 1 < a.d_v && pairs) {
                    *reinterpret_cast<uint32_t*>(dst + c) =
                        pack_pair(o[j][2 * hh] * scale * gate_16(__uint_as_float(g2[j] << 16), a.gate_act),
                                  o[j][2 * hh + 1] * scale * gate_16(__uint_as_float(g2[j] & 0xffff0000u), a.gate_act));
                } else {
                    for (int e = 0; e < 2; ++e)
                        if (c + e < a.d_v)
                            dst[c + e] = __float2bfloat16_rn(o[j][2 * hh + e] * scale * gate_16(__bfloat162float(gate[c + e]), a.gate_act));
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

static size_t outputs_smem(int d_k, int ns, int parts) {
    const int d_pad = (d_k + 15) / 16 * 16;
    return sizeof(__nv_bfloat16) * ((size_t)2 * parts * kRun * (d_pad + 8) + (size_t)kRun * (ns + 8) + (size_t)2 * d_pad * (ns + 8));
}
static size_t sums_smem(int d_k, int ns) {
    const int d_pad = (d_k + 15) / 16 * 16;
    return sizeof(__nv_bfloat16) * ((size_t)2 * kRun * (d_pad + 8) + (size_t)kRun * (ns + 8));
}
constexpr size_t kMostSmem = 227 * 1024 - 1024;    // (a kilobyte for the static part)

// columns of the values a CTA takes: all of a head's up to 128 where shared memory allows, else slices of 64; 0: no fit
static int run_columns(int d_k, int d_v) {
    if (d_v > 64 && outputs_smem(d_k, 128, 2) <= kMostSmem) return 128;
    return outputs_smem(d_k, 64, 2) <= kMostSmem ? 64 : 0;
}

template <int NS, int PARTS>
static int launch_runs(const FixedDecayArgs& a, int n_seqs, int max_q_len, cudaStream_t stream) {
    const size_t s1 = sums_smem(a.d_k, NS), s3 = outputs_smem(a.d_k, NS, PARTS);
    static size_t have1 = 48 * 1024, have3 = 48 * 1024;
    if (s1 > have1) {
        const int e = (int)cudaFuncSetAttribute(fixed_decay_run_sums_kernel<NS, PARTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        if (e != 0) return e;
        have1 = s1;
    }
    if (s3 > have3) {
        const int e = (int)cudaFuncSetAttribute(fixed_decay_outputs_kernel<NS, PARTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
        if (e != 0) return e;
        have3 = s3;
    }
    const int n_runs = (max_q_len + kRun - 1) / kRun, slices = (a.d_v + NS - 1) / NS;
    const dim3 grid(n_runs * slices, a.heads, n_seqs);
    int st = launch_pdl(fixed_decay_run_sums_kernel<NS, PARTS>, grid, dim3(kRunThreads), s1, stream, a);
    if (st != 0) return st;
    st = launch_pdl(fixed_decay_carry_kernel, dim3((a.d_k * a.d_v + 255) / 256, a.heads, n_seqs), dim3(256), 0, stream, a);
    if (st != 0) return st;
    return launch_pdl(fixed_decay_outputs_kernel<NS, PARTS>, grid, dim3(kRunThreads), s3, stream, a);
}

// Whether queries and keys, and values, can be read as they lie, or a kernel has to leave them on the run kernels' grid first.
static bool qk_ready(const FixedDecayArgs& a) {
    return !a.qk_silu && a.pairs == 0 && a.d_k % 16 == 0 && a.ld_q % 8 == 0 && a.ld_k % 8 == 0 && (((uintptr_t)a.q | (uintptr_t)a.k) & 15) == 0;
}
static bool v_ready(const FixedDecayArgs& a) {
    return !a.v_silu && a.d_v % 8 == 0 && a.ld_v % 8 == 0 && ((uintptr_t)a.v & 15) == 0;
}
static size_t run_floats(int n_tokens, int n_seqs, int heads, int d_k, int d_v) {   // of the runs' sums, to a multiple of 4
    return (((size_t)(n_tokens / kRun + n_seqs + 1) * heads * d_k * d_v) + 3) / 4 * 4;
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
// Floats of scratch the prompt kernels need: the runs' sums, then queries, keys and values in the run kernels' layout.
extern "C" long long b200_fixed_decay_scratch(int n_tokens, int n_seqs, int heads, int d_k, int d_v) {
    const long long d_pad = (d_k + 15) / 16 * 16, v_pad = (d_v + 7) / 8 * 8;
    return (long long)b200::run_floats(n_tokens, n_seqs, heads, d_k, d_v) + ((4 * d_pad + v_pad) * n_tokens * heads + 1) / 2;
}

// The recurrence over a packed step (see the head of this file).  n_tokens == n_seqs: one token per sequence, operands of
// either type; otherwise bfloat16 operands and `scratch` as b200_fixed_decay_scratch says.
// out: float32 [T, heads d_v], or rows (not null): the finished heads, o / rms(o) * act(gate) * mul, into [T, ld_rows].
extern "C" int b200_fixed_decay(const void* q, int ld_q, const void* k, int ld_k, const void* v, int ld_v, const float* decay,
                                float* state, long long slot_stride, const int* slots, const int* cu_seqlens, const int* positions,
                                const float* inv_freq, int pairs, float* out, float* scratch, int dtype,
                                int n_tokens, int n_seqs, int max_q_len, int heads, int d_k, int d_v, float q_scale, int qk_silu,
                                int v_silu, const void* gate, int ld_gate, int gate_act, void* rows, int ld_rows, float eps, float mul,
                                cudaStream_t stream) {
    using namespace b200;
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (heads < 1 || heads > 65535 || n_seqs > 65535 || d_k < 1 || d_v < 1 || d_k > 512 || pairs < 0 || 2 * pairs > d_k || !decay)
        return kErrBadArgument;
    if ((rows == nullptr) == (out == nullptr) || (rows != nullptr && (!gate || ld_rows < heads * d_v || ld_gate < heads * d_v)))
        return kErrBadArgument;
    if (pairs > 0 && (!inv_freq || !positions)) return kErrBadArgument;
    FixedDecayArgs a = {};
    a.q = q; a.k = k; a.v = v; a.ld_q = ld_q; a.ld_k = ld_k; a.ld_v = ld_v;
    a.decay = decay; a.state = state; a.slot_stride = (size_t)slot_stride; a.slots = slots; a.cu_seqlens = cu_seqlens;
    a.inv_freq = inv_freq; a.positions = positions; a.out = out; a.runs = scratch;
    a.n_tokens = n_tokens; a.heads = heads; a.d_k = d_k; a.d_v = d_v; a.pairs = pairs; a.qk_silu = qk_silu; a.v_silu = v_silu;
    a.q_scale = q_scale; a.gate = gate; a.ld_gate = ld_gate; a.gate_act = gate_act; a.rows = rows; a.ld_rows = ld_rows; a.eps = eps; a.mul = mul;
    if (n_tokens == n_seqs) {
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
    if (!scratch || ((uintptr_t)scratch & 15)) return kErrBadArgument;
    // queries and keys have two parts where they are turned (32-bit numbers), one where they are projections
    const int parts = pairs > 0 ? 2 : 1;
    PrepareRows prep = {};
    prep.d_pad = (d_k + 15) / 16 * 16;
    prep.v_pad = (d_v + 7) / 8 * 8;
    __nv_bfloat16* room = reinterpret_cast<__nv_bfloat16*>(scratch + run_floats(n_tokens, n_seqs, heads, d_k, d_v));
    const size_t qk_size = (size_t)n_tokens * heads * prep.d_pad;
    a.qt[0] = (const __nv_bfloat16*)q; a.kt[0] = (const __nv_bfloat16*)k; a.vt = (const __nv_bfloat16*)v;
    a.ld_qt = ld_q; a.ld_kt = ld_k; a.ld_vt = ld_v; a.head_qk = d_k; a.head_v = d_v;
    if (!qk_ready(a)) {
        for (int w = 0; w < 2; ++w)
            for (int p = 0; p < parts; ++p) prep.qk[w][p] = room + (size_t)(2 * w + p) * qk_size;
        for (int p = 0; p < parts; ++p) { a.qt[p] = prep.qk[0][p]; a.kt[p] = prep.qk[1][p]; }
        a.ld_qt = a.ld_kt = heads * prep.d_pad;
        a.head_qk = prep.d_pad;
    }
    if (!v_ready(a)) {
        prep.v = room + 4 * qk_size;
        a.vt = prep.v;
        a.ld_vt = heads * prep.v_pad;
        a.head_v = prep.v_pad;
    }
    if (prep.qk[0][0] != nullptr || prep.v != nullptr) {
        const int st = launch_pdl(fixed_decay_prepare_kernel, dim3(n_tokens), dim3(128), sizeof(float) * 2 * pairs, stream, a, prep);
        if (st != 0) return st;
    }
    if (ns == 128) return parts == 2 ? launch_runs<128, 2>(a, n_seqs, max_q_len, stream) : launch_runs<128, 1>(a, n_seqs, max_q_len, stream);
    return parts == 2 ? launch_runs<64, 2>(a, n_seqs, max_q_len, stream) : launch_runs<64, 1>(a, n_seqs, max_q_len, stream);
}
