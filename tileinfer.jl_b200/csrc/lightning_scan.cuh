// The scan of a step's tokens through a matrix state per (sequence, head), S_t = a S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, as a template
// over what happens to q, k, the decay and the input on the way (MODE, below). Included by the files that launch it, one per mode.
#pragma once
#include "common.cuh"

#define LS_COLS 32
#define LS_TOKENS 32
#define LS_MAX_DIM 512

__device__ __forceinline__ float silu_value(float z) { return z / (1.0f + expf(-z)); }

// What a scan does beyond the plain recurrence.
//   MODE 0   nothing: q, k, v through the activation, one decay per head
//   MODE 1   the first `rotary` elements of every q and k head are rotated by the token's position (element i with i + rotary / 2;
//            cos_sin [positions, rotary / 2, 2]; null: no rotation), then q and k are multiplied by q_scale and k_scale
//   MODE 2   S_t = keep_t S_(t-1) + add_t k_t v_t^T with coef [tokens, heads, 2] = (keep, add) per token, and beside S a vector
//            n_t = keep_t n_(t-1) + add_t k_t [dim] per head (it lies H * D * V floats into the sequence's state), whose product n_t . q_t
//            goes to nq [tokens, heads]: n is one more column of S whose value is always one, and its column blocks are launched
//            after the V columns'. q and k are multiplied by q_scale and k_scale.
// A token's row of o has H * V floats; a sequence's state lies at slot * state_stride floats.
struct ScanExtras {
    long long state_stride;
    const float* cos_sin;
    int rotary;
    const int* positions;
    float q_scale, k_scale;
    const float* coef;
    float* nq;
};

template <typename T, int DP, bool VECTORS, int LS_PARTS, int MODE>
__global__ void __launch_bounds__(LS_COLS* LS_PARTS) lightning_scan_kernel(
    float* __restrict__ o, const T* qkv, long long ld, int q_off, int k_off, int v_off, float* state,
    const float* __restrict__ decay, const int* cu_seqlens, const int* seq_slots, int H, int D, int V, int act, int split, ScanExtras ex) {
    extern __shared__ float smem[];
    float* qs = smem;                                   // [LS_TOKENS][D]
    float* ks = qs + LS_TOKENS * D;                     // [LS_TOKENS][D]
    float* vs = ks + LS_TOKENS * D;                     // [LS_TOKENS][LS_COLS]
    float* part = vs + LS_TOKENS * LS_COLS;             // [LS_TOKENS][LS_PARTS][LS_COLS]
    __shared__ float keeps[MODE == 2 ? LS_TOKENS : 1], adds[MODE == 2 ? LS_TOKENS : 1];
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    // With `split` > 1 the rows of S are shared out among that many blocks, whose shares of o are added up in global memory.
    const int col0 = (blockIdx.x / split) * LS_COLS, h = blockIdx.y, b = blockIdx.z;
    const int rows_per = (D + split - 1) / split, row0 = (blockIdx.x % split) * rows_per, row1 = min(D, row0 + rows_per);
    const int col = col0 + lane;
    const float a0 = MODE == 2 ? 1.f : decay[h];
    const int v_end = MODE == 2 ? V + 1 : V;            // columns of the state, the vector n counted as one
    pdl_enter();
    const int t0 = __ldcg(cu_seqlens + b), t1 = __ldcg(cu_seqlens + b + 1);
    const int slot = __ldcg(seq_slots + b);
    float* S = state + (size_t)slot * ex.state_stride + (size_t)h * D * V;
    const bool is_n = MODE == 2 && col == V;            // this lane's column is the vector n
    float* mine = is_n ? state + (size_t)slot * ex.state_stride + (size_t)H * D * V + (size_t)h * D : S + col;
    const size_t pitch = is_n ? 1 : V;
    float s[DP];
#pragma unroll
    for (int i = 0; i < DP; ++i) {
        const int d = row0 + w * DP + i;
        s[i] = (d < row1 && col < v_end) ? __ldcg(mine + (size_t)d * pitch) : 0.f;
    }
    // The rows of a batch of 16 tokens come in 16-byte vectors where the layout allows it, and the next batch's are asked for
    // before this batch's arithmetic, so that their way from memory is hidden behind it.
    constexpr int VEC = 16 / (int)sizeof(T), MAXV = 4;
    const bool wide = VECTORS && D % VEC == 0 && V % VEC == 0;
    const int qk_vecs = D / VEC;                        // vectors in a head's row of q (and of k)
    constexpr int V_VECS = LS_COLS / VEC;               // vectors in the block's 32 columns of v
    uint4 rq[MAXV], rk[MAXV], rv;
    auto fetch = [&](int base, int count) {
#pragma unroll
        for (int i = 0; i < MAXV; ++i) {
            const int idx = threadIdx.x + i * (LS_COLS * LS_PARTS);
            if (idx < count * qk_vecs) {
                const T* row = qkv + (size_t)(base + idx / qk_vecs) * ld + (size_t)h * D + (idx % qk_vecs) * VEC;
                rq[i] = __ldcg(reinterpret_cast<const uint4*>(row + q_off));
                rk[i] = __ldcg(reinterpret_cast<const uint4*>(row + k_off));
            }
        }
        const int idx = threadIdx.x;
        if (idx < count * V_VECS && col0 + (idx % V_VECS) * VEC < V)
            rv = __ldcg(reinterpret_cast<const uint4*>(qkv + (size_t)(base + idx / V_VECS) * ld + v_off + (size_t)h * V + col0 + (idx % V_VECS) * VEC));
    };
    auto put = [&](float* dst, const uint4& raw, float scale) {
        Vec16<T> v;
        if constexpr (sizeof(T) == 2) v.unpack(raw);
        else { v.v[0] = __uint_as_float(raw.x); v.v[1] = __uint_as_float(raw.y); v.v[2] = __uint_as_float(raw.z); v.v[3] = __uint_as_float(raw.w); }
#pragma unroll
        for (int e = 0; e < VEC; ++e)           // (16-bit rows: the fast exponential and division are far below their rounding)
            dst[e] = MODE != 0 ? v.v[e] * scale : !act ? v.v[e] : sizeof(T) == 2 ? rnd<T>(__fdividef(v.v[e], 1.0f + __expf(-v.v[e]))) : silu_value(v.v[e]);
    };
    if (wide && t0 < t1) fetch(t0, min(LS_TOKENS, t1 - t0));
    for (int base = t0; base < t1; base += LS_TOKENS) {
        const int count = min(LS_TOKENS, t1 - base);
        // (No barrier here: every thread has passed the barrier after the last batch's arithmetic, so its rows may be
        // overwritten; the shares of o that slow threads may still be adding up are rewritten only after the next barrier.)
        if (wide) {
#pragma unroll
            for (int i = 0; i < MAXV; ++i) {
                const int idx = threadIdx.x + i * (LS_COLS * LS_PARTS);
                if (idx < count * qk_vecs) {
                    put(qs + (idx / qk_vecs) * D + (idx % qk_vecs) * VEC, rq[i], ex.q_scale);
                    put(ks + (idx / qk_vecs) * D + (idx % qk_vecs) * VEC, rk[i], ex.k_scale);
                }
            }
            const int idx = threadIdx.x;
            if (idx < count * V_VECS) {
                float* dst = vs + (idx / V_VECS) * LS_COLS + (idx % V_VECS) * VEC;
                if (col0 + (idx % V_VECS) * VEC < V) put(dst, rv, 1.f);
                else
#pragma unroll
                    for (int e = 0; e < VEC; ++e) dst[e] = MODE == 2 && col0 + (idx % V_VECS) * VEC + e == V ? 1.f : 0.f;
            }
            if (base + LS_TOKENS < t1) fetch(base + LS_TOKENS, min(LS_TOKENS, t1 - base - LS_TOKENS));
        } else {
        for (int e = threadIdx.x; e < count * D; e += blockDim.x) {
            const int t = e / D, d = e % D;
            const T* row = qkv + (size_t)(base + t) * ld + (size_t)h * D + d;
            float qv = to_f32(__ldcg(row + q_off)), kv = to_f32(__ldcg(row + k_off));
            if (MODE != 0) { qv *= ex.q_scale; kv *= ex.k_scale; }
            else if (act) { qv = rnd<T>(silu_value(qv)); kv = rnd<T>(silu_value(kv)); }
            qs[t * D + d] = qv;
            ks[t * D + d] = kv;
        }
        for (int e = threadIdx.x; e < count * LS_COLS; e += blockDim.x) {
            const int t = e / LS_COLS, c = e % LS_COLS;
            float vv = 0.f;
            if (col0 + c < V) {
                vv = to_f32(__ldcg(qkv + (size_t)(base + t) * ld + v_off + (size_t)h * V + col0 + c));
                if (MODE == 0 && act) vv = rnd<T>(silu_value(vv));
            } else if (MODE == 2 && col0 + c == V) vv = 1.f;
            vs[t * LS_COLS + c] = vv;
        }
        }
        if (MODE == 2 && threadIdx.x < count) {
            const float2 c2 = __ldcg(reinterpret_cast<const float2*>(ex.coef) + (size_t)(base + threadIdx.x) * H + h);
            keeps[threadIdx.x] = c2.x;
            adds[threadIdx.x] = c2.y;
        }
        __syncthreads();
        if (MODE == 1 && ex.cos_sin != nullptr) {
            // The pairs of every head in place (the scales, the same for both elements of a pair, are already in).
            const int half = ex.rotary >> 1, p0 = __ldcg(ex.positions + base);          // a sequence's tokens are consecutive
            for (int e = threadIdx.x; e < count * half; e += blockDim.x) {
                const int t = e / half, i = e - t * half;
                const float2 cs = __ldg(reinterpret_cast<const float2*>(ex.cos_sin) + (size_t)(p0 + t) * half + i);
                float* qt = qs + t * D + i;
                float* kt = ks + t * D + i;
                const float qu = qt[0], qv = qt[half], ku = kt[0], kv = kt[half];
                qt[0] = qu * cs.x - qv * cs.y; qt[half] = qv * cs.x + qu * cs.y;
                kt[0] = ku * cs.x - kv * cs.y; kt[half] = kv * cs.x + ku * cs.y;
            }
            __syncthreads();
        }
        // One token: the state's rows of this warp move on and give their share of o. Four partial sums keep the chain of
        // dependent additions short; the order of a token's sum still depends on the sizes alone.
        auto token = [&](int t) {
            const float a = MODE == 2 ? keeps[t] : a0;
            const float vt = MODE == 2 ? vs[t * LS_COLS + lane] * adds[t] : vs[t * LS_COLS + lane];
            const float* qt = qs + t * D;
            const float* kt = ks + t * D;
            float acc0 = 0.f, acc1 = 0.f, acc2 = 0.f, acc3 = 0.f;
            if (D % 4 == 0 && rows_per % 4 == 0) {       // (DP is a multiple of 4: four rows' k and q per shared-memory read)
#pragma unroll
                for (int i = 0; i < DP; i += 4) {
                    const int d = row0 + w * DP + i;
                    if (d < row1) {
                        const float4 k4 = *reinterpret_cast<const float4*>(kt + d), q4 = *reinterpret_cast<const float4*>(qt + d);
                        s[i] = fmaf(a, s[i], k4.x * vt); acc0 = fmaf(s[i], q4.x, acc0);
                        s[i + 1] = fmaf(a, s[i + 1], k4.y * vt); acc1 = fmaf(s[i + 1], q4.y, acc1);
                        s[i + 2] = fmaf(a, s[i + 2], k4.z * vt); acc2 = fmaf(s[i + 2], q4.z, acc2);
                        s[i + 3] = fmaf(a, s[i + 3], k4.w * vt); acc3 = fmaf(s[i + 3], q4.w, acc3);
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < DP; ++i) {
                    const int d = row0 + w * DP + i;
                    if (d < row1) {
                        s[i] = fmaf(a, s[i], kt[d] * vt);
                        acc0 = fmaf(s[i], qt[d], acc0);
                    }
                }
            }
            part[(t * LS_PARTS + w) * LS_COLS + lane] = (acc0 + acc1) + (acc2 + acc3);
        };
        if (count == LS_TOKENS) {
#pragma unroll 4
            for (int t = 0; t < LS_TOKENS; ++t) token(t);
        } else {
            for (int t = 0; t < count; ++t) token(t);
        }
        __syncthreads();
        for (int e = threadIdx.x; e < count * LS_COLS; e += blockDim.x) {
            const int t = e / LS_COLS, c = e % LS_COLS;
            if (col0 + c >= v_end) continue;
            float sum = 0.f;
#pragma unroll
            for (int p = 0; p < LS_PARTS; ++p) sum += part[(t * LS_PARTS + p) * LS_COLS + c];
            float* dst = MODE == 2 && col0 + c == V ? ex.nq + (size_t)(base + t) * H + h : o + (size_t)(base + t) * H * V + (size_t)h * V + col0 + c;
            if (split > 1) atomicAdd(dst, sum);         // o was zeroed; with two addends the sum does not depend on their order
            else *dst = sum;
        }
    }
#pragma unroll
    for (int i = 0; i < DP; ++i) {
        const int d = row0 + w * DP + i;
        if (d < row1 && col < v_end) mine[(size_t)d * pitch] = s[i];
    }
}

// Launches the scan for `n_tokens` tokens of B sequences; the arguments are those of the kernel.
template <int MODE>
static int launch_lightning_scan(const char* what, float* o, const void* qkv, long long ld, int q_off, int k_off, int v_off, float* state,
                                 const float* decay, const int* cu_seqlens, const int* seq_slots, int n_tokens, int B, int H, int D, int V, int act,
                                 const ScanExtras& ex, int dtype, cudaStream_t stream) {
    TI_REQUIRE(H > 0 && D > 0 && V > 0 && D <= LS_MAX_DIM, "%s: %d heads of %d x %d (the key size is at most %d)", what, H, D, V, LS_MAX_DIM);
    TI_REQUIRE(H <= 65535 && B <= 65535, "%s: %d heads, %d sequences", what, H, B);
    // A launch with few blocks (one prompt of a model with few heads) shares the rows of S out between two blocks each.
    const int col_blocks = ((MODE == 2 ? V + 1 : V) + LS_COLS - 1) / LS_COLS;
    const int split = ((long long)col_blocks * H * B < 100 && D >= 16) ? 2 : 1;
    if (split > 1 && cudaMemsetAsync(o, 0, (size_t)n_tokens * H * V * sizeof(float), stream) != cudaSuccess) return ti_fail("%s: memset failed", what);
    if (split > 1 && MODE == 2 && cudaMemsetAsync(ex.nq, 0, (size_t)n_tokens * H * sizeof(float), stream) != cudaSuccess) return ti_fail("%s: memset failed", what);
    const dim3 grid(col_blocks * split, H, B);
    // Few blocks walking long sequences are bound by latency: 16 warps a block then (each with half the rows); many blocks, or
    // one-token steps, which are bound by reading and writing the state, run better with 8.
    const int parts = ((long long)col_blocks * split * H * B <= 160 && n_tokens >= 64 * B) ? 16 : 8;
    const size_t smem = (size_t)(2 * LS_TOKENS * D + LS_TOKENS * LS_COLS + LS_TOKENS * parts * LS_COLS) * sizeof(float);
    const int dp = ((D + split - 1) / split + parts - 1) / parts;
    // 16-byte loads need every row's pieces on 16-byte borders and at most four vectors of q per thread and batch of tokens.
#define LS_LAUNCH2(DP, PARTS)                                                                                                        \
    do {                                                                                                                             \
        constexpr int VEC = 16 / (int)sizeof(T);                                                                                     \
        const bool vectors = aligned16(qkv) && ld % VEC == 0 && q_off % VEC == 0 && k_off % VEC == 0 && v_off % VEC == 0 &&          \
                             LS_TOKENS * (D / VEC) <= 4 * LS_COLS * PARTS;                                                           \
        if (smem > 40 * 1024) {                                                                                                      \
            cudaFuncSetAttribute(lightning_scan_kernel<T, DP, true, PARTS, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            cudaFuncSetAttribute(lightning_scan_kernel<T, DP, false, PARTS, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        }                                                                                                                            \
        if (vectors)                                                                                                                 \
            ti_launch(lightning_scan_kernel<T, DP, true, PARTS, MODE>, grid, dim3(LS_COLS* PARTS), smem, stream, o, (const T*)qkv, ld, q_off, k_off,    \
                      v_off, state, decay, cu_seqlens, seq_slots, H, D, V, act, split, ex);                                              \
        else                                                                                                                         \
            ti_launch(lightning_scan_kernel<T, DP, false, PARTS, MODE>, grid, dim3(LS_COLS* PARTS), smem, stream, o, (const T*)qkv, ld, q_off, k_off,   \
                      v_off, state, decay, cu_seqlens, seq_slots, H, D, V, act, split, ex);                                              \
    } while (0)
#define LS_LAUNCH(DP)                        \
    do {                                     \
        if (parts == 16) LS_LAUNCH2(DP, 16); \
        else LS_LAUNCH2(DP, 8);              \
    } while (0)
    TI_DISPATCH_DTYPE(dtype, {
        if (dp <= 4) LS_LAUNCH(4);
        else if (dp <= 8) LS_LAUNCH(8);
        else if (dp <= 16) LS_LAUNCH(16);
        else if (dp <= 32) LS_LAUNCH(32);
        else LS_LAUNCH(64);
    });
#undef LS_LAUNCH2
#undef LS_LAUNCH
    return ti_check_launch(what);
}
