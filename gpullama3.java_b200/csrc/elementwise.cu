// Small per-element and per-row kernels that several parts share.
//   softcap_rows       x <- cap * tanh(x / cap), in place on 32-bit logits
//   gated_rmsnorm      out[t, h, :] = x[t, h, :] / sqrt(mean(x^2) + eps) * w * act(gate[t, h, :]), act sigmoid or SiLU
//                      per (token, head) row of 32-bit numbers: the output norm of a recurrent mixer; with `gate_first`
//                      the row is multiplied by act(gate) first and the norm runs over the gated row; with
//                      `weight_per_row` every row has weights of its own (w holds n_heads * d numbers), so that the rows
//                      may be any equal parts of the mixer's output, not its heads; a warp per row, or a CTA per row
//                      of 512 numbers and more; w may be absent, `mul` is a last factor, and the output's rows may be
//                      columns of a wider buffer
//   turn_back_rows     out[t, h, :d] = mul * (x[t, h, :d] turned by -position * inv_freq over the row's halves): the results of
//                      attention over values that were cached turned by their own positions; x's heads are d_pad wide,
//                      the output's rows may be columns of a wider buffer; a CTA per token, angles once per token
//   gate_rows          x[t, :n] <- x[t, :n] * sigmoid(gate[t, :n]) (or SiLU), in place: a gate on a mixer's output
//   scale_rows         x <- x * s, in place on 32-bit logits
//   differential_heads out[t, h, :] = post * o / sqrt(mean(o^2) + eps) * sigmoid(gate[t, h, :]) with o = a1 - lambda a2, where
//                      a1 and a2 are the results of two attention maps over the same values that lie as neighbouring
//                      heads (2h, 2h + 1) of `d_pad` numbers of which the first `d` count; a warp per (token, head)
#include "common.cuh"

namespace b200 {

__global__ void softcap_kernel(float* __restrict__ x, size_t n, float cap) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] / cap);
}

// a warp per (token, head) row
template <typename T>
__global__ void __launch_bounds__(128)
gated_rmsnorm_kernel(const float* __restrict__ x, const float* __restrict__ w, const T* __restrict__ gate, int ld_gate,
                     T* __restrict__ out, int ld_out, float mul, int n_heads, int d, int n_rows, float eps, int gate_act, int gate_first,
                     int weight_per_row) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= n_rows) return;
    const int t = row / n_heads, h = row % n_heads;
    const float* xr = x + (size_t)row * d;
    const T* g = gate + (size_t)t * ld_gate + (size_t)h * d;
    const float* wr = w ? w + (weight_per_row ? (size_t)h * d : 0) : nullptr;
    auto weight = [&](int e) { return wr ? wr[e] : 1.f; };
    auto act = [&](int e) {
        const float z = to_f32<T>(g[e]);
        const float sig = 1.0f / (1.0f + expf(-z));
        return gate_act == 1 ? z * sig : sig;
    };
    float ss = 0.f;
    for (int e = lane; e < d; e += 32) {
        const float v = gate_first ? xr[e] * act(e) : xr[e];
        ss += v * v;
    }
    ss = warp_sum(ss);
    const float scale = mul / sqrtf(ss / (float)d + eps);
    T* o = out + (size_t)t * ld_out + (size_t)h * d;
    for (int e = lane; e < d; e += 32)
        o[e] = from_f32<T>(gate_first ? (xr[e] * act(e)) * scale * weight(e) : xr[e] * scale * weight(e) * act(e));
}

// a CTA per row, for rows too long for one warp (a norm over a large part of the mixer's output); the gated values stay
// in registers between the two passes when the row has at most kWideKeep * VEC numbers per thread.  VEC 4: 16-byte accesses of
// the row and the weight, where sizes and pointers allow.
constexpr int kWideThreads = 256, kWideKeep = 8;
template <typename T, int VEC> __device__ __forceinline__ void load_row(const T* p, float (&f)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) f[e] = to_f32<T>(p[e]);
}
template <> __device__ __forceinline__ void load_row<float, 4>(const float* p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
template <> __device__ __forceinline__ void load_row<__nv_bfloat16, 4>(const __nv_bfloat16* p, float (&f)[4]) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
}
template <typename T, int VEC> __device__ __forceinline__ void store_row(T* p, const float (&f)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) p[e] = from_f32<T>(f[e]);
}
template <> __device__ __forceinline__ void store_row<float, 4>(float* p, const float (&f)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
template <> __device__ __forceinline__ void store_row<__nv_bfloat16, 4>(__nv_bfloat16* p, const float (&f)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kWideThreads)
gated_rmsnorm_wide_kernel(const float* __restrict__ x, const float* __restrict__ w, const T* __restrict__ gate, int ld_gate,
                          T* __restrict__ out, int ld_out, float mul, int n_heads, int d, float eps, int gate_act, int gate_first,
                          int weight_per_row) {
    __shared__ float scratch[33];
    constexpr int kKeep = VEC == 4 ? 2 : kWideKeep, kStep = kWideThreads * VEC;
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x;
    const int t = row / n_heads, h = row % n_heads;
    const float* xr = x + (size_t)row * d;
    const T* g = gate + (size_t)t * ld_gate + (size_t)h * d;
    const float* wr = w ? w + (weight_per_row ? (size_t)h * d : 0) : nullptr;
    // a piece of VEC numbers from column e on, multiplied by its gate where the gate comes first; `a` holds the gate otherwise
    auto piece = [&](int e, float (&v)[VEC], float (&a)[VEC]) {
        load_row<float, VEC>(xr + e, v);
        load_row<T, VEC>(g + e, a);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float sig = 1.0f / (1.0f + expf(-a[i]));
            a[i] = gate_act == 1 ? a[i] * sig : sig;
            if (gate_first) { v[i] *= a[i]; a[i] = 1.f; }
        }
    };
    float keep[kKeep][VEC], act[kKeep][VEC], ss = 0.f;
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
        const int e = threadIdx.x * VEC + i * kStep;
        if (e < d) {
            piece(e, keep[i], act[i]);
#pragma unroll
            for (int c = 0; c < VEC; ++c) ss += keep[i][c] * keep[i][c];
        }
    }
    for (int e = threadIdx.x * VEC + kKeep * kStep; e < d; e += kStep) {
        float v[VEC], a[VEC];
        piece(e, v, a);
#pragma unroll
        for (int c = 0; c < VEC; ++c) ss += v[c] * v[c];
    }
    ss = block_sum(ss, scratch);
    const float scale = mul / sqrtf(ss / (float)d + eps);
    T* o = out + (size_t)t * ld_out + (size_t)h * d;
    auto finish = [&](int e, float (&v)[VEC], const float (&a)[VEC]) {
        float wv[VEC];
#pragma unroll
        for (int c = 0; c < VEC; ++c) wv[c] = 1.f;
        if (wr) load_row<float, VEC>(wr + e, wv);
#pragma unroll
        for (int c = 0; c < VEC; ++c) v[c] = v[c] * scale * wv[c] * a[c];
        store_row<T, VEC>(o + e, v);
    };
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
        const int e = threadIdx.x * VEC + i * kStep;
        if (e < d) finish(e, keep[i], act[i]);
    }
    for (int e = threadIdx.x * VEC + kKeep * kStep; e < d; e += kStep) {
        float v[VEC], a[VEC];
        piece(e, v, a);
        finish(e, v, a);
    }
}

template <typename T>
__global__ void gate_rows_kernel(T* __restrict__ x, int ld_x, const T* __restrict__ gate, int ld_gate, int n, int gate_act) {
    T* xr = x + (size_t)blockIdx.x * ld_x;
    const T* g = gate + (size_t)blockIdx.x * ld_gate;
    for (int e = blockIdx.y * blockDim.x + threadIdx.x; e < n; e += gridDim.y * blockDim.x) {
        const float z = to_f32<T>(g[e]);
        const float sig = 1.0f / (1.0f + expf(-z));
        xr[e] = from_f32<T>(to_f32<T>(xr[e]) * (gate_act == 1 ? z * sig : sig));
    }
}

template <typename T>
__global__ void __launch_bounds__(128)
differential_heads_kernel(const T* __restrict__ maps, const T* __restrict__ gate, int ld_gate, T* __restrict__ out, int ld_out,
                          int n_heads, int d, int d_pad, int n_rows, float lambda, float post, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= n_rows) return;
    const int t = row / n_heads, h = row % n_heads;
    const T* a1 = maps + ((size_t)row * 2) * d_pad;
    const T* a2 = a1 + d_pad;
    float ss = 0.f;
    for (int e = lane; e < d; e += 32) {
        const float o = to_f32<T>(a1[e]) - lambda * to_f32<T>(a2[e]);
        ss += o * o;
    }
    ss = warp_sum(ss);
    const float scale = post / sqrtf(ss / (float)d + eps);
    const T* g = gate ? gate + (size_t)t * ld_gate + (size_t)h * d : nullptr;
    T* o_row = out + (size_t)t * ld_out + (size_t)h * d;
    for (int e = lane; e < d; e += 32) {
        float o = (to_f32<T>(a1[e]) - lambda * to_f32<T>(a2[e])) * scale;
        if (g) o *= 1.0f / (1.0f + expf(-to_f32<T>(g[e])));
        o_row[e] = from_f32<T>(o);
    }
}

// VEC neighbouring pairs per thread (4: 8-byte accesses of 16-bit numbers, where sizes and pointers allow)
constexpr int kTurnThreads = 128, kTurnPairs = 256;
template <typename T, int VEC> struct TurnVec {
    __device__ static void load(const T* p, float (&f)[VEC]) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) f[e] = to_f32<T>(p[e]);
    }
    __device__ static void store(T* p, const float (&f)[VEC]) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) p[e] = from_f32<T>(f[e]);
    }
};
template <> struct TurnVec<__nv_bfloat16, 4> {
    __device__ static void load(const __nv_bfloat16* p, float (&f)[4]) {
        const uint2 v = *reinterpret_cast<const uint2*>(p);
        f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
        f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
    }
    __device__ static void store(__nv_bfloat16* p, const float (&f)[4]) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    }
};
template <typename T, int VEC>
__global__ void __launch_bounds__(kTurnThreads)
turn_back_rows_kernel(const T* __restrict__ x, const int* __restrict__ positions, const float* __restrict__ inv_freq,
                      T* __restrict__ out, int ld_out, int n_heads, int d, int d_pad, float mul) {
    __shared__ float cos_s[kTurnPairs], sin_s[kTurnPairs];
    pdl_launch_dependents();
    const int t = blockIdx.x, n = d / 2;
    // positions were copied in before the step's first kernel: the angles are made before the wait
    const float pos = inv_freq ? (float)positions[t] : 0.f;
    for (int i = threadIdx.x; i < n && inv_freq; i += kTurnThreads) sincosf(pos * inv_freq[i], &sin_s[i], &cos_s[i]);
    __syncthreads();
    pdl_wait();
    const T* xr = x + (size_t)t * n_heads * d_pad;
    T* o = out + (size_t)t * ld_out;
    if (!inv_freq) {
        for (int u = blockIdx.y * kTurnThreads + threadIdx.x; u < n_heads * d; u += gridDim.y * kTurnThreads)
            o[u] = from_f32<T>(to_f32<T>(xr[(size_t)(u / d) * d_pad + u % d]) * mul);
        return;
    }
    const int per_head = n / VEC;
    for (int u = blockIdx.y * kTurnThreads + threadIdx.x; u < n_heads * per_head; u += gridDim.y * kTurnThreads) {
        const int h = u / per_head, i = (u % per_head) * VEC;
        float a[VEC], b[VEC];
        TurnVec<T, VEC>::load(xr + (size_t)h * d_pad + i, a);
        TurnVec<T, VEC>::load(xr + (size_t)h * d_pad + i + n, b);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float c = cos_s[i + e], s = sin_s[i + e], p = a[e], q = b[e];
            a[e] = (p * c + q * s) * mul;
            b[e] = (q * c - p * s) * mul;
        }
        TurnVec<T, VEC>::store(o + (size_t)h * d + i, a);
        TurnVec<T, VEC>::store(o + (size_t)h * d + i + n, b);
    }
}

__global__ void scale_kernel(float* __restrict__ x, size_t n, float s) {
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) x[i] *= s;
}

}  // namespace b200

extern "C" int b200_softcap_rows(float* x, long long n, float cap, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (!(cap > 0.f)) return b200::kErrBadArgument;
    const long long blocks = (n + 255) / 256;
    b200::softcap_kernel<<<(int)(blocks < 148 * 16 ? blocks : 148 * 16), 256, 0, stream>>>(x, (size_t)n, cap);
    return b200::launch_status();
}

extern "C" int b200_gated_rmsnorm(const float* x, const float* w, const void* gate, int ld_gate, void* out, int dtype,
                                  int n_tokens, int n_heads, int d, float eps, int gate_act, int gate_first,
                                  int weight_per_row, int ld_out, float mul, cudaStream_t stream) {
    if (gate_act != 0 && gate_act != 1) return b200::kErrBadArgument;   // 0 sigmoid, 1 SiLU
    if (n_tokens <= 0 || n_heads <= 0) return 0;
    if (d < 1 || ld_out < n_heads * d) return b200::kErrBadArgument;
    const long long rows = (long long)n_tokens * n_heads;
    if (rows > 0x7fffffffLL) return b200::kErrUnsupportedSize;
    const size_t el = dtype == b200::kF32 ? 4 : 2;
    const bool wide4 = d % 4 == 0 && ld_gate % 4 == 0 && ld_out % 4 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0 &&
                       ((uintptr_t)gate % (4 * el)) == 0 && ((uintptr_t)out % (4 * el)) == 0;
    B200_DISPATCH_DTYPE(dtype, T,
        if (d >= 512) {    // (a warp would walk such a row in 16 or more rounds, twice)
            if (wide4)
                return b200::launch_pdl(b200::gated_rmsnorm_wide_kernel<T, 4>, dim3((unsigned)rows), dim3(b200::kWideThreads), 0, stream, x, w,
                                        (const T*)gate, ld_gate, (T*)out, ld_out, mul, n_heads, d, eps, gate_act, gate_first, weight_per_row);
            return b200::launch_pdl(b200::gated_rmsnorm_wide_kernel<T, 1>, dim3((unsigned)rows), dim3(b200::kWideThreads), 0, stream, x, w,
                                    (const T*)gate, ld_gate, (T*)out, ld_out, mul, n_heads, d, eps, gate_act, gate_first, weight_per_row);
        }
        return b200::launch_pdl(b200::gated_rmsnorm_kernel<T>, dim3((unsigned)((rows + 3) / 4)), dim3(128), 0, stream, x, w, (const T*)gate,
                                ld_gate, (T*)out, ld_out, mul, n_heads, d, (int)rows, eps, gate_act, gate_first, weight_per_row));
    return b200::launch_status();
}

extern "C" int b200_gate_rows(void* x, int ld_x, const void* gate, int ld_gate, int dtype, int n_tokens, int n, int gate_act,
                              cudaStream_t stream) {
    if (gate_act != 0 && gate_act != 1) return b200::kErrBadArgument;
    if (n_tokens <= 0 || n <= 0) return 0;
    const int ny = (n + 1023) / 1024;
    B200_DISPATCH_DTYPE(dtype, T,
        b200::gate_rows_kernel<T><<<dim3(n_tokens, ny > 64 ? 64 : ny), 256, 0, stream>>>((T*)x, ld_x, (const T*)gate, ld_gate, n,
                                                                                        gate_act));
    return b200::launch_status();
}

extern "C" int b200_scale_rows(float* x, long long n, float s, cudaStream_t stream) {
    if (n <= 0) return 0;
    const long long blocks = (n + 255) / 256;
    b200::scale_kernel<<<(int)(blocks < 148 * 16 ? blocks : 148 * 16), 256, 0, stream>>>(x, (size_t)n, s);
    return b200::launch_status();
}

// maps [T][2 n_heads][d_pad], gate [T][ld_gate] (or null), out [T][ld_out >= n_heads d], all of the run's type
extern "C" int b200_differential_heads(const void* maps, const void* gate, int ld_gate, void* out, int ld_out, int dtype, int n_tokens,
                                       int n_heads, int d, int d_pad, float lambda, float post, float eps,
                                       cudaStream_t stream) {
    if (n_tokens <= 0 || n_heads <= 0) return 0;
    if (d < 1 || d_pad < d || ld_out < n_heads * d || (gate && ld_gate < n_heads * d)) return b200::kErrBadArgument;
    const long long rows = (long long)n_tokens * n_heads;
    if (rows > 0x7fffffffLL) return b200::kErrUnsupportedSize;
    B200_DISPATCH_DTYPE(dtype, T,
        return b200::launch_pdl(b200::differential_heads_kernel<T>, dim3((int)((rows + 3) / 4)), dim3(128), 0, stream,
                                (const T*)maps, (const T*)gate, ld_gate, (T*)out, ld_out, n_heads, d, d_pad, (int)rows, lambda, post, eps));
    return 0;
}

// x [T][n_heads d_pad], out [T][ld_out >= n_heads d] of the run's type; d even; inv_freq float32 [d / 2] (null: nothing is
// turned, the heads are only moved and scaled)
extern "C" int b200_turn_back_rows(const void* x, const int* positions, const float* inv_freq, void* out, int ld_out, int dtype,
                                   int n_tokens, int n_heads, int d, int d_pad, float mul, cudaStream_t stream) {
    if (n_tokens <= 0 || n_heads <= 0) return 0;
    if (d < 1 || d_pad < d || ld_out < n_heads * d || (inv_freq && (d % 2 || !positions))) return b200::kErrBadArgument;
    if (inv_freq && d / 2 > b200::kTurnPairs) return b200::kErrUnsupportedSize;
    const bool vec = inv_freq && d % 8 == 0 && d_pad % 4 == 0 && ld_out % 4 == 0 && (((uintptr_t)x | (uintptr_t)out) & 7) == 0 && dtype == b200::kBF16;
    const int units = n_heads * (inv_freq ? d / 2 : d) / (vec ? 4 : 1);
    int ny = n_tokens >= 512 ? 1 : (units + b200::kTurnThreads - 1) / b200::kTurnThreads;   // few tokens: a token's heads over several CTAs
    if (ny > 64) ny = 64;
    B200_DISPATCH_DTYPE(dtype, T,
        if (vec)
            return b200::launch_pdl(b200::turn_back_rows_kernel<T, 4>, dim3(n_tokens, ny), dim3(b200::kTurnThreads), 0, stream, (const T*)x,
                                    positions, inv_freq, (T*)out, ld_out, n_heads, d, d_pad, mul);
        return b200::launch_pdl(b200::turn_back_rows_kernel<T, 1>, dim3(n_tokens, ny), dim3(b200::kTurnThreads), 0, stream, (const T*)x,
                                positions, inv_freq, (T*)out, ld_out, n_heads, d, d_pad, mul));
    return 0;
}
