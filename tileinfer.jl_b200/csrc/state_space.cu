// The state-space recurrence of Mamba-2 around its matrix memory: per head h, with one decay and one step size per token,
//
//   S_t = e^(l_t) S_(t-1) + dt_t B_t x_t^T     [state, vdim]        y_t = S_t^T C_t + D_h x_t
//   dt = softplus(dt' + dt_bias_h),  l = -exp(A_log_h) dt           heads of a group share B and C
//
//   ssm_inputs      the projected rows [z | x | B | C | dt']: x, B and C through a causal convolution over time with a bias and SiLU,
//                   rounded once; (l, dt) of every token and head in 32-bit. In one-token steps the convolution's history moves on as
//                   well (a thread owns its channels); otherwise history_update does, a launch of its own
//   ssm_token       one token per sequence: the state read and written once
//   ssm_gate_norm   (y silu(z)), the row in equal parts, each divided by its own root mean square, times a weight
//
// Steps of several tokens per sequence go through memory_chunks.cu. The state, (l, dt) and everything computed from them are 32-bit.
#include "common.cuh"

#define SI_MAX_TAPS 16
#define SI_TOKENS 16             // rows a block walks in steps of several tokens per sequence
#define SI_AHEAD 4               // rows whose loads are in flight together

__device__ __forceinline__ float ssm_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ssm_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <typename T, int VEC> struct Cells {           // VEC neighbouring elements of T or of float
    static __device__ __forceinline__ void load(const T* p, float (&v)[VEC]) {
        if constexpr (VEC == 4 && sizeof(T) == 2) {
            const uint2 t = __ldcg(reinterpret_cast<const uint2*>(p));
            v[0] = __uint_as_float(t.x << 16); v[1] = __uint_as_float(t.x & 0xffff0000u);
            v[2] = __uint_as_float(t.y << 16); v[3] = __uint_as_float(t.y & 0xffff0000u);
        } else if constexpr (VEC == 4) {
            const float4 t = __ldcg(reinterpret_cast<const float4*>(p));
            v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
        } else {
            v[0] = to_f32(__ldcg(p));
        }
    }
    static __device__ __forceinline__ void store(T* p, const float (&v)[VEC]) {
        if constexpr (VEC == 4 && sizeof(T) == 2) {
            const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
            *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&a), *reinterpret_cast<const unsigned*>(&b));
        } else if constexpr (VEC == 4) {
            *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        } else {
            p[0] = from_f32<T>(v[0]);
        }
    }
};

struct SsmInputs {
    long long ld;                // elements between rows
    int x_off, dt_off, C, H;     // first column of x | B | C (C channels) and of dt' (H)
    int taps;
    float* hist;                 // [slots][taps - 1][C] float, hist_stride floats a slot
    long long hist_stride;
    const float* dt_bias;        // [H]
    const float* a_log;          // [H]
    const int* cu_seqlens;
    const int* seq_slots;
    int B, n, decode, tokens;    // tokens: rows of a block
};

// Blocks (channels, `tokens` rows), and one more column of blocks for (l, dt). conv is [taps][C].
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(128) ssm_inputs_kernel(T* __restrict__ xbc, float* __restrict__ coef, const T* rows, const T* __restrict__ conv,
                                                         const T* __restrict__ bias, SsmInputs a) {
    const int first = blockIdx.y * a.tokens, last = min(a.n, first + a.tokens);
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    const int ntaps = TAPS > 0 ? TAPS : a.taps;
    constexpr int SLOTS = TAPS > 0 ? TAPS : 1, BACK = TAPS > 1 ? TAPS - 1 : 1;
    float c[SLOTS][VEC], w[BACK][VEC], bc[VEC];
    const bool channels = blockIdx.x + 1 < gridDim.x;
    if (channels && i < a.C) {
        if (TAPS > 0)
#pragma unroll
            for (int j = 0; j < TAPS; ++j) Cells<T, VEC>::load(conv + (size_t)j * a.C + i, c[j]);
        Cells<T, VEC>::load(bias + i, bc);
    }
    pdl_enter();
    if (!channels) {
        for (int e = threadIdx.x; e < (last - first) * a.H; e += blockDim.x) {
            const int t = first + e / a.H, h = e % a.H;
            const float dt = ssm_softplus(to_f32(__ldcg(rows + (size_t)t * a.ld + a.dt_off + h)) + a.dt_bias[h]);
            reinterpret_cast<float2*>(coef)[(size_t)t * a.H + h] = make_float2(-expf(a.a_log[h]) * dt, dt);
        }
        return;
    }
    if (i >= a.C) return;
    int lo = 0, hi = a.B - 1;                            // the sequence of the first row: the last b with cu[b] <= first
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (__ldcg(a.cu_seqlens + mid) <= first) lo = mid; else hi = mid - 1;
    }
    int b = lo, begin = __ldcg(a.cu_seqlens + b), end = __ldcg(a.cu_seqlens + b + 1);
    const T* src = rows + a.x_off + i;
    auto earlier = [&](int r, float (&u)[VEC]) {         // row r of the step, or, ahead of the sequence's first, a row of its history
        if (r >= begin) Cells<T, VEC>::load(src + (size_t)r * a.ld, u);
        else Cells<float, VEC>::load(a.hist + (size_t)__ldcg(a.seq_slots + b) * a.hist_stride + (size_t)(ntaps - 1 - (begin - r)) * a.C + i, u);
    };
    auto finish = [&](int t, float (&acc)[VEC]) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float z = acc[e] + bc[e];              // (16-bit rows: the fast exponential and division are far below their rounding)
            acc[e] = sizeof(T) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : ssm_silu(z);
        }
        Cells<T, VEC>::store(xbc + (size_t)t * a.C + i, acc);
    };
    bool fresh = true;                                   // the rows before the current one are not in registers
    int t = first;
    while (t < last) {
        while (t >= end) { ++b; begin = __ldcg(a.cu_seqlens + b); end = __ldcg(a.cu_seqlens + b + 1); fresh = true; }
        if (TAPS > 0) {
            const int rows_now = min(SI_AHEAD, min(last, end) - t);
            float u[SI_AHEAD][VEC];
#pragma unroll
            for (int q = 0; q < SI_AHEAD; ++q)
                if (q < rows_now) Cells<T, VEC>::load(src + (size_t)(t + q) * a.ld, u[q]);
            if (TAPS > 1 && fresh)
#pragma unroll
                for (int j = 0; j < BACK; ++j) earlier(t - BACK + j, w[j]);
            fresh = false;
#pragma unroll
            for (int q = 0; q < SI_AHEAD; ++q) {
                if (q >= rows_now) break;
                float acc[VEC];
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) acc[e] = fmaf(c[j][e], w[j][e], acc[e]);
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[e] = fmaf(c[SLOTS - 1][e], u[q][e], acc[e]);
                if (a.decode && TAPS > 1) {              // one token per sequence: these channels' history moves up by one row
                    float* st = a.hist + (size_t)__ldcg(a.seq_slots + b) * a.hist_stride + i;
#pragma unroll
                    for (int j = 0; j + 1 < BACK; ++j) Cells<float, VEC>::store(st + (size_t)j * a.C, w[j + 1]);
                    Cells<float, VEC>::store(st + (size_t)(BACK - 1) * a.C, u[q]);
                }
#pragma unroll
                for (int j = 0; j + 1 < BACK; ++j)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) w[j][e] = w[j + 1][e];
#pragma unroll
                for (int e = 0; e < VEC; ++e) w[BACK - 1][e] = u[q][e];
                finish(t + q, acc);
            }
            t += rows_now;
        } else {
            float u[VEC], acc[VEC];
            Cells<T, VEC>::load(src + (size_t)t * a.ld, u);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
            float* st = a.hist + (size_t)__ldcg(a.seq_slots + b) * a.hist_stride + i;
            for (int j = 0; j < ntaps; ++j) {
                float v[VEC], cj[VEC];
                if (j + 1 < ntaps) earlier(t - (ntaps - 1) + j, v);
                Cells<T, VEC>::load(conv + (size_t)j * a.C + i, cj);
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[e] = fmaf(cj[e], j + 1 < ntaps ? v[e] : u[e], acc[e]);
                if (a.decode && j > 0) Cells<float, VEC>::store(st + (size_t)(j - 1) * a.C, j + 1 < ntaps ? v : u);
            }
            finish(t, acc);
            ++t;
        }
    }
}

// rows [n, ld] of T; conv [taps][C] and bias [C] of T; xbc [n, C] of T; coef [n, H, 2] float = (l, dt). decode: one token per sequence,
// the history moves on.
extern "C" int ti_ssm_inputs(void* xbc, float* coef, const void* rows, long long ld, int x_off, int dt_off, const void* conv, int taps, const void* bias,
                             float* hist, long long hist_stride, const float* dt_bias, const float* a_log, const int* cu_seqlens, const int* seq_slots,
                             int n, int B, int C, int H, int decode, int dtype, cudaStream_t stream) {
    if (n == 0) return 0;
    TI_REQUIRE(taps >= 1 && taps <= SI_MAX_TAPS && (taps == 1 || hist != nullptr) && C > 0 && H > 0 && B > 0, "ssm_inputs: %d taps, %d channels, %d heads", taps, C, H);
    const SsmInputs a = {ld, x_off, dt_off, C, H, taps, hist, hist_stride, dt_bias, a_log, cu_seqlens, seq_slots, B, n, decode, decode ? 1 : SI_TOKENS};
#define SI_LAUNCH(V, TAPS) ti_launch(ssm_inputs_kernel<T, V, TAPS>, grid, dim3(128), 0, stream, (T*)xbc, coef, (const T*)rows, (const T*)conv, (const T*)bias, a)
#define SI_TAPS(V)                        \
    switch (taps) {                       \
        case 1: SI_LAUNCH(V, 1); break;   \
        case 2: SI_LAUNCH(V, 2); break;   \
        case 3: SI_LAUNCH(V, 3); break;   \
        case 4: SI_LAUNCH(V, 4); break;   \
        default: SI_LAUNCH(V, 0); break;  \
    }
    TI_DISPATCH_DTYPE(dtype, {
        const uintptr_t mask = sizeof(T) == 2 ? 7 : 15;
        const bool vec = C % 4 == 0 && ld % 4 == 0 && x_off % 4 == 0 && hist_stride % 4 == 0 && aligned16(hist) &&
                         (((uintptr_t)xbc | (uintptr_t)rows | (uintptr_t)conv | (uintptr_t)bias) & mask) == 0;
        const dim3 grid((vec ? C / 4 + 127 : C + 127) / 128 + 1, (n + a.tokens - 1) / a.tokens);
        if (vec) { SI_TAPS(4) } else { SI_TAPS(1) }
    });
#undef SI_TAPS
#undef SI_LAUNCH
    return ti_check_launch("ssm_inputs");
}

// ------------------------------------------------------------------------------------------------ one token per sequence
#define ST_THREADS 256
// A block owns one (sequence, head) and up to 256 pieces of VEC columns of its state: a thread owns one piece and takes every `per`-th row,
// eight rows' loads in flight; the rows' shares of y meet in shared memory.
template <typename T, int VEC>
__global__ void __launch_bounds__(ST_THREADS) ssm_token_kernel(float* __restrict__ y, const T* xbc, const float* coef, const float* __restrict__ skip,
                                                               float* state, long long state_stride, const int* seq_slots, int C, int H, int heads_per_group,
                                                               int N, int V, int b_off, int c_off) {
    extern __shared__ __align__(16) float smem[];
    const int h = blockIdx.y, b = blockIdx.z, g = h / heads_per_group;
    const int pieces = min(ST_THREADS, V / VEC - (int)blockIdx.x * ST_THREADS), per = ST_THREADS / pieces;
    float* bs = smem;                                    // [N]
    float* cs = bs + (N + 3) / 4 * 4;                    // [N]
    float* part = cs + (N + 3) / 4 * 4;                  // [per][pieces * VEC]
    const int piece = threadIdx.x % pieces, row0 = threadIdx.x / pieces, col = (blockIdx.x * ST_THREADS + piece) * VEC;
    pdl_enter();
    float* S = state + (size_t)__ldcg(seq_slots + b) * state_stride + (size_t)h * N * V + col;
    const bool works = row0 < per;
    constexpr int U = 8;
    float s[U][VEC];
    auto fetch = [&](int d0) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int d = d0 + u * per;
            if (d < N) Cells<float, VEC>::load(S + (size_t)d * V, s[u]);
        }
    };
    if (works) fetch(row0);
    const T* row = xbc + (size_t)b * C;
    for (int d = threadIdx.x; d < N; d += ST_THREADS) {
        bs[d] = to_f32(__ldcg(row + b_off + (size_t)g * N + d));
        cs[d] = to_f32(__ldcg(row + c_off + (size_t)g * N + d));
    }
    const float2 co = __ldcg(reinterpret_cast<const float2*>(coef) + (size_t)b * H + h);
    const float keep = expf(co.x);
    float x[VEC], acc[VEC];
    Cells<T, VEC>::load(row + (size_t)h * V + col, x);
#pragma unroll
    for (int e = 0; e < VEC; ++e) { x[e] *= co.y; acc[e] = 0.f; }
    __syncthreads();
    if (works) {
        for (int d0 = row0; d0 < N; d0 += U * per) {
            if (d0 != row0) fetch(d0);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int d = d0 + u * per;
                if (d < N) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        s[u][e] = fmaf(keep, s[u][e], bs[d] * x[e]);
                        acc[e] = fmaf(s[u][e], cs[d], acc[e]);
                    }
                    Cells<float, VEC>::store(S + (size_t)d * V, s[u]);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) part[(row0 * pieces + piece) * VEC + e] = acc[e];
    }
    __syncthreads();
    for (int c = threadIdx.x; c < pieces * VEC; c += ST_THREADS) {
        float sum = 0.f;
        for (int p = 0; p < per; ++p) sum += part[p * pieces * VEC + c];
        const int v = blockIdx.x * ST_THREADS * VEC + c;
        y[(size_t)b * H * V + (size_t)h * V + v] = fmaf(skip[h], to_f32(__ldcg(row + (size_t)h * V + v)), sum);
    }
}

// xbc [B, C] of T: x (H * V columns), B (groups * N) from b_off on, C from c_off on; coef [B, H, 2]; a sequence's state [H, N, V] float at
// slot * state_stride; y [B, H * V] float.
extern "C" int ti_ssm_token(float* y, const void* xbc, const float* coef, const float* skip, float* state, long long state_stride, const int* seq_slots,
                            int B, int C, int H, int groups, int N, int V, int dtype, cudaStream_t stream) {
    if (B == 0) return 0;
    TI_REQUIRE(H > 0 && groups > 0 && H % groups == 0 && N > 0 && V > 0 && N <= 4096 && H <= 65535 && B <= 65535, "ssm_token: %d heads in %d groups, %d x %d", H, groups, N, V);
    const int b_off = H * V, c_off = b_off + groups * N;
    TI_DISPATCH_DTYPE(dtype, {
        const bool vec = V % 4 == 0 && C % 4 == 0 && state_stride % 4 == 0 && aligned16(state) && (((uintptr_t)xbc) & (sizeof(T) == 2 ? 7 : 15)) == 0;
        const int v = vec ? 4 : 1, blocks = (V / v + ST_THREADS - 1) / ST_THREADS;
        const size_t smem = (size_t)(2 * ((N + 3) / 4 * 4) + ST_THREADS * v) * sizeof(float);
        if (vec) ti_launch(ssm_token_kernel<T, 4>, dim3(blocks, H, B), dim3(ST_THREADS), smem, stream, y, (const T*)xbc, coef, skip, state, state_stride, seq_slots, C, H, H / groups, N, V, b_off, c_off);
        else ti_launch(ssm_token_kernel<T, 1>, dim3(blocks, H, B), dim3(ST_THREADS), smem, stream, y, (const T*)xbc, coef, skip, state, state_stride, seq_slots, C, H, H / groups, N, V, b_off, c_off);
    });
    return ti_check_launch("ssm_token");
}

// ------------------------------------------------------------------------------------------------ gate, then norm in parts
// out [n, size] of T = (y silu(z)) / rms(over each of `parts` equal parts) * w. A block per row; `team` warps share a part where there
// are fewer parts than warps. The order of a part's sum depends on the sizes alone.
template <typename T, int VEC>
__global__ void ssm_gate_norm_kernel(T* __restrict__ out, const float* y, const T* z, long long ldz, const T* __restrict__ w, float eps, int parts, int size) {
    extern __shared__ __align__(16) float row[];         // [size], then [parts], then partial sums
    float* inv = row + (size + 3) / 4 * 4;
    float* sums = inv + parts;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    pdl_enter();
    for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
        float v[VEC], g[VEC];
        Cells<float, VEC>::load(y + (size_t)blockIdx.x * size + i, v);
        Cells<T, VEC>::load(z + (size_t)blockIdx.x * ldz + i, g);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] *= ssm_silu(g[e]);
        Cells<float, VEC>::store(row + i, v);
    }
    __syncthreads();
    const int per = size / parts, team = warps > parts ? warps / parts : 1, teams = warps / team;
    if (warp < teams * team)
        for (int q = warp / team; q < parts; q += teams) {
            float ss = 0.f;
            for (int i = (warp % team) * 32 + lane; i < per; i += team * 32) ss = fmaf(row[q * per + i], row[q * per + i], ss);
            ss = warp_sum(ss);
            if (lane == 0) sums[q * team + warp % team] = ss;
        }
    __syncthreads();
    for (int q = threadIdx.x; q < parts; q += blockDim.x) {
        float ss = 0.f;
        for (int p = 0; p < team; ++p) ss += sums[q * team + p];
        inv[q] = 1.0f / sqrtf(ss / (float)per + eps);
    }
    __syncthreads();
    for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
        float v[VEC], wv[VEC];
        Cells<T, VEC>::load(w + i, wv);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = row[i + e] * inv[(i + e) / per] * wv[e];
        Cells<T, VEC>::store(out + (size_t)blockIdx.x * size + i, v);
    }
}

extern "C" int ti_ssm_gate_norm(void* out, const float* y, const void* z, long long ldz, const void* w, float eps, int parts, int n, int size, int dtype,
                                cudaStream_t stream) {
    if (n == 0) return 0;
    TI_REQUIRE(size > 0 && parts >= 1 && parts <= 4096 && size % parts == 0 && size <= 40000, "ssm_gate_norm: rows of %d in %d parts", size, parts);
    const int threads = size >= 4096 ? 512 : size >= 1024 ? 256 : 128;
    const size_t smem = (size_t)((size + 3) / 4 * 4 + parts + (parts > threads / 32 ? parts : threads / 32)) * sizeof(float);
    TI_DISPATCH_DTYPE(dtype, {
        const bool vec = size % 4 == 0 && ldz % 4 == 0 && aligned16(y) && (((uintptr_t)out | (uintptr_t)z | (uintptr_t)w) & (sizeof(T) == 2 ? 7 : 15)) == 0;
        if (smem > 48 * 1024) {
            cudaFuncSetAttribute(ssm_gate_norm_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            cudaFuncSetAttribute(ssm_gate_norm_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        }
        if (vec) ti_launch(ssm_gate_norm_kernel<T, 4>, dim3(n), dim3(threads), smem, stream, (T*)out, y, (const T*)z, ldz, (const T*)w, eps, parts, size);
        else ti_launch(ssm_gate_norm_kernel<T, 1>, dim3(n), dim3(threads), smem, stream, (T*)out, y, (const T*)z, ldz, (const T*)w, eps, parts, size);
    });
    return ti_check_launch("ssm_gate_norm");
}
