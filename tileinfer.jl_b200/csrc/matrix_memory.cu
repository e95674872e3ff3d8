// A matrix memory per (sequence, head) with exponential gates kept in range by a running maximum (the mLSTM cell of xLSTM), and the
// one-token step that it shares with retention.
//
//   i = cap tanh((zi + bi) / cap),  f = log sigmoid(cap tanh((zf + bf) / cap)),  m_t = max(f + m_(t-1), i)         one per token and head
//   keep = exp(f + m_(t-1) - m_t),  add = exp(i - m_t)
//   S_t = keep S_(t-1) + add k v^T,  n_t = keep n_(t-1) + add k,  o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)
//
//   memory_gates   i, f and m of every token of the step as a scan of the block's tokens (t maps m to max(m + f_t, i_t), and such maps
//                  compose), then keep, add and exp(-m)
//   memory_scan    the recurrence over a step's tokens (lightning_scan.cuh, MODE 2); the division is left to heads_norm_gate
//   memory_token   one token per sequence, for this cell and for retention: rotation or gates, the state read and written once, and,
//                  where a block holds a whole head, its RMS norm, weight and output gate as well
//
// A sequence's state is one block of floats: S [H, dim, vdim], n [H, dim], m [H] (retention: S alone). All of it is 32-bit.
#include "lightning_scan.cuh"

#define MG_THREADS 256
#define MEMORY_FLOOR 1e-6f

__device__ __forceinline__ float capped_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

__global__ void __launch_bounds__(MG_THREADS) memory_gates_kernel(float* __restrict__ coef, float* __restrict__ em, const float* z, long long ldz,
                                                                  const float* __restrict__ bias, float cap, float* m_state,
                                                                  long long state_stride, const int* cu_seqlens, const int* seq_slots, int H) {
    __shared__ float tf[MG_THREADS / 32], ti[MG_THREADS / 32], last;
    const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    const float bi = bias[h], bf = bias[H + h];
    pdl_enter();
    const int t0 = __ldcg(cu_seqlens + b), t1 = __ldcg(cu_seqlens + b + 1);
    float* slot_m = m_state + (size_t)__ldcg(seq_slots + b) * state_stride + h;
    float m = __ldcg(slot_m);
    for (int base = t0; base < t1; base += MG_THREADS) {
        const int t = base + threadIdx.x;
        const bool in = t < t1;
        float gi = -INFINITY, gf = 0.f;                  // a token that is not there leaves m as it is
        if (in) {
            gi = capped_gate(__ldcg(z + (size_t)t * ldz + h) + bi, cap);
            gf = log_sigmoid(capped_gate(__ldcg(z + (size_t)t * ldz + H + h) + bf, cap));
        }
        float F = gf, I = gi;                            // this token's map, then that of all tokens of the warp up to it
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pf = __shfl_up_sync(0xffffffffu, F, o), pi = __shfl_up_sync(0xffffffffu, I, o);
            if (lane >= o) { I = fmaxf(pi + F, I); F += pf; }
        }
        if (lane == 31) { tf[w] = F; ti[w] = I; }
        __syncthreads();
        float before = m;                                // m ahead of the warp's first token
        for (int v = 0; v < w; ++v) before = fmaxf(before + tf[v], ti[v]);
        const float mt = fmaxf(before + F, I);
        float prev = __shfl_up_sync(0xffffffffu, mt, 1);
        if (lane == 0) prev = before;
        if (in) {
            reinterpret_cast<float2*>(coef)[(size_t)t * H + h] = make_float2(expf(gf + prev - mt), expf(gi - mt));
            em[(size_t)t * H + h] = expf(-mt);
            if (t == min(base + MG_THREADS, t1) - 1) last = mt;
        }
        __syncthreads();
        m = last;
    }
    if (threadIdx.x == 0 && t0 < t1) *slot_m = m;
}

// coef [n, H, 2] and em [n, H] float for the step's tokens; z [n, ldz] float: the logits of i (H of them), then of f; bias [2 H];
// m_state: where head 0's m lies in slot 0's state. m moves on to the step's last token.
extern "C" int ti_memory_gates(float* coef, float* em, const float* z, long long ldz, const float* bias, float cap, float* m_state,
                               long long state_stride, const int* cu_seqlens, const int* seq_slots, int B, int H, cudaStream_t stream) {
    if (B == 0) return 0;
    TI_REQUIRE(H > 0 && B <= 65535 && cap > 0.f, "memory_gates: %d heads, %d sequences, cap %g", H, B, cap);
    ti_launch(memory_gates_kernel, dim3(H, B), dim3(MG_THREADS), 0, stream, coef, em, z, ldz, bias, cap, m_state, state_stride, cu_seqlens, seq_slots, H);
    return ti_check_launch("memory_gates");
}

// o [n, H * V] (not yet divided) and nq [n, H] = n . q, float.
extern "C" int ti_memory_scan(float* o, float* nq, const void* qkv, long long ld, int q_off, int k_off, int v_off, float* state, long long state_stride,
                              const float* coef, float q_scale, float k_scale, const int* cu_seqlens, const int* seq_slots, int n_tokens, int B, int H,
                              int D, int V, int dtype, cudaStream_t stream) {
    if (B == 0) return 0;
    ScanExtras ex = {};
    ex.state_stride = state_stride;
    ex.q_scale = q_scale; ex.k_scale = k_scale;
    ex.coef = coef; ex.nq = nq;
    return launch_lightning_scan<2>("memory_scan", o, qkv, ld, q_off, k_off, v_off, state, nullptr, cu_seqlens, seq_slots, n_tokens, B, H, D, V, 0, ex,
                                    dtype, stream);
}

// ------------------------------------------------------------------------------------------------ one token per sequence
#define MT_WARPS 8
struct TokenExtras {
    // retention: one decay per head, an optional rotation
    const float* decay;
    const float* cos_sin;
    int rotary;
    const int* positions;
    // the gated cell (z not null): gate logits [B, ldz] with their biases [2 H]
    const float* z;
    long long ldz;
    const float* bias;
    float cap;
    float q_scale, k_scale;
    // the head's output, where a block holds the whole head
    const void* w;           // [H * V] of T or null
    int g_off;               // column of the output gate's logits in the rows
    int gate_sigmoid;        // the gate's activation: sigmoid, or SiLU
    float eps;
    // what the next kernel needs, where it does not
    float* nq;               // [B, H]
    float* em;               // [B, H]
    float* m_new;            // [B, H]
};

// A block owns 128 columns of one (sequence, head): a lane owns four of them (16 bytes of a row), the warps take the rows in turn, and
// their shares of o meet in shared memory.
template <typename T>
__global__ void __launch_bounds__(MT_WARPS * 32) memory_token_kernel(T* __restrict__ y, float* __restrict__ o, const T* qkv, long long ld, int q_off, int k_off,
                                                                     int v_off, float* state, long long state_stride, const int* seq_slots, int H,
                                                                     int D, int V, TokenExtras ex) {
    extern __shared__ float smem[];
    float* qs = smem;                                   // [D]
    float* ks = qs + D;                                 // [D]
    float* part = ks + ((D + 3) / 4 * 4 - D) * 2 + D;   // [MT_WARPS][128], on a 16-byte border
    __shared__ float scratch[33], gates[3];             // gates: keep, add, m
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, threads = MT_WARPS * 32;
    const int col = blockIdx.x * 128 + lane * 4, h = blockIdx.y, b = blockIdx.z;
    const bool gated = ex.z != nullptr;
    pdl_enter();
    float* base = state + (size_t)__ldcg(seq_slots + b) * state_stride;
    float* S = base + (size_t)h * D * V;
    const T* row = qkv + (size_t)b * ld;
    if (gated && threadIdx.x == 0) {
        const float i = capped_gate(__ldcg(ex.z + (size_t)b * ex.ldz + h) + ex.bias[h], ex.cap);
        const float f = log_sigmoid(capped_gate(__ldcg(ex.z + (size_t)b * ex.ldz + H + h) + ex.bias[H + h], ex.cap));
        const float m_old = __ldcg(base + (size_t)H * D * V + (size_t)H * D + h), m = fmaxf(f + m_old, i);
        gates[0] = expf(f + m_old - m); gates[1] = expf(i - m); gates[2] = m;
    }
    const int half = ex.rotary >> 1;
    const float2* cs = ex.cos_sin != nullptr ? reinterpret_cast<const float2*>(ex.cos_sin) + (size_t)__ldcg(ex.positions + b) * half : nullptr;
    for (int d = threadIdx.x; d < D; d += threads) {
        const T* q = row + q_off + (size_t)h * D;
        const T* k = row + k_off + (size_t)h * D;
        float qv = to_f32(__ldcg(q + d)) * ex.q_scale, kv = to_f32(__ldcg(k + d)) * ex.k_scale;
        if (cs != nullptr && d < ex.rotary) {
            const int i = d < half ? d : d - half, other = d < half ? d + half : d - half;
            const float2 c = __ldg(cs + i);
            const float sign = d < half ? -1.f : 1.f;
            const float qo = to_f32(__ldcg(q + other)) * ex.q_scale, ko = to_f32(__ldcg(k + other)) * ex.k_scale;
            qv = qv * c.x + sign * (qo * c.y);
            kv = kv * c.x + sign * (ko * c.y);
        }
        qs[d] = qv;
        ks[d] = kv;
    }
    float v4[4] = {0.f, 0.f, 0.f, 0.f};
    if (col < V) {
#pragma unroll
        for (int e = 0; e < 4; ++e) v4[e] = to_f32(__ldcg(row + v_off + (size_t)h * V + col + e));
    }
    __syncthreads();
    const float a = gated ? gates[0] : ex.decay[h];
    if (gated) {
#pragma unroll
        for (int e = 0; e < 4; ++e) v4[e] *= gates[1];
    }
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (col < V) {
#pragma unroll 8
        for (int d = w; d < D; d += MT_WARPS) {
            float4 s4 = __ldcg(reinterpret_cast<const float4*>(S + (size_t)d * V + col));
            const float kd = ks[d], qd = qs[d];
            s4.x = fmaf(a, s4.x, kd * v4[0]); s4.y = fmaf(a, s4.y, kd * v4[1]);
            s4.z = fmaf(a, s4.z, kd * v4[2]); s4.w = fmaf(a, s4.w, kd * v4[3]);
            acc[0] = fmaf(s4.x, qd, acc[0]); acc[1] = fmaf(s4.y, qd, acc[1]);
            acc[2] = fmaf(s4.z, qd, acc[2]); acc[3] = fmaf(s4.w, qd, acc[3]);
            *reinterpret_cast<float4*>(S + (size_t)d * V + col) = s4;
        }
    }
    *reinterpret_cast<float4*>(part + w * 128 + lane * 4) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    float nq = 0.f, em = 0.f;
    if (gated && blockIdx.x == 0) {                     // the vector n: one block of the head
        float* n = base + (size_t)H * D * V + (size_t)h * D;
        float share = 0.f;
        for (int d = threadIdx.x; d < D; d += threads) {
            const float v = fmaf(a, __ldcg(n + d), ks[d] * gates[1]);
            n[d] = v;
            share = fmaf(v, qs[d], share);
        }
        nq = block_sum(share, scratch);
        em = expf(-gates[2]);
    }
    __syncthreads();
    const int c = threadIdx.x;                          // (128 columns, 256 threads)
    float sum = 0.f;
    const bool mine = c < 128 && blockIdx.x * 128 + c < V;
    if (mine) {
#pragma unroll
        for (int p = 0; p < MT_WARPS; ++p) sum += part[p * 128 + c];
    }
    if (y == nullptr) {
        if (mine) o[(size_t)b * H * V + (size_t)h * V + blockIdx.x * 128 + c] = sum;
        if (gated && blockIdx.x == 0 && threadIdx.x == 0) {
            ex.nq[(size_t)b * H + h] = nq;
            ex.em[(size_t)b * H + h] = em;
            ex.m_new[(size_t)b * H + h] = gates[2];
        }
        return;
    }
    if (gated) {
        sum /= fmaxf(fabsf(nq), em) + MEMORY_FLOOR;
        if (threadIdx.x == 0) base[(size_t)H * D * V + (size_t)H * D + h] = gates[2];
    }
    const float inv = 1.0f / sqrtf(block_sum(mine ? sum * sum : 0.f, scratch) / (float)V + ex.eps);
    if (mine) {
        const float g = to_f32(__ldcg(row + ex.g_off + (size_t)h * V + c));
        float v = sum * inv;
        if (ex.w != nullptr) v *= to_f32(reinterpret_cast<const T*>(ex.w)[(size_t)h * V + c]);
        v *= (ex.gate_sigmoid ? 1.0f : g) / (1.0f + expf(-g));
        y[(size_t)b * H * V + (size_t)h * V + c] = from_f32<T>(v);
    }
}

// Returns 2 when the sizes are outside what this kernel takes (then a one-token step runs through the scan). Give `y` [B, H * V] for
// heads of up to 128 values (the whole mixer output before the output projection), else `o` [B, H * V] float with, for the gated
// cell, nq, em and m_new [B, H].
extern "C" int ti_memory_token(void* y, float* o, float* nq, float* em, float* m_new, const void* qkv, long long ld, int q_off, int k_off, int v_off,
                               int g_off, float* state, long long state_stride, const float* decay, const float* z, long long ldz, const float* bias,
                               float cap, const float* cos_sin, int rotary, const int* positions, float q_scale, float k_scale, const void* w,
                               int gate_sigmoid, float eps, const int* seq_slots, int B, int H, int D, int V, int dtype, cudaStream_t stream) {
    if (B == 0) return 0;
    TI_REQUIRE((decay != nullptr) != (z != nullptr) && (y != nullptr) != (o != nullptr), "memory_token: one decay per head or gates, y or o");
    TI_REQUIRE(y == nullptr || V <= 128, "memory_token: a head of %d values is shared out between blocks", V);
    TI_REQUIRE(z == nullptr || (bias != nullptr && cap > 0.f && (o == nullptr || (nq != nullptr && em != nullptr && m_new != nullptr))),
               "memory_token: the gated cell needs its biases, a cap and its outputs");
    TI_REQUIRE(cos_sin == nullptr || (positions != nullptr && rotary >= 2 && rotary % 2 == 0 && rotary <= D), "memory_token: rotation over %d of %d", rotary, D);
    if (V % 4 != 0 || state_stride % 4 != 0 || !aligned16(state) || D > 2048 || H > 65535 || B > 65535) {
        ti_fail("memory_token takes value sizes in steps of 4 and key sizes up to 2048; got %d x %d", D, V);
        return 2;
    }
    const TokenExtras ex = {decay, cos_sin, cos_sin != nullptr ? rotary : 0, positions, z, ldz, bias, cap, q_scale, k_scale, w, g_off, gate_sigmoid, eps, nq, em, m_new};
    const size_t smem = (size_t)(2 * ((D + 3) / 4 * 4) + MT_WARPS * 128) * sizeof(float);
    TI_DISPATCH_DTYPE(dtype, (ti_launch(memory_token_kernel<T>, dim3((V + 127) / 128, H, B), dim3(MT_WARPS * 32), smem, stream, (T*)y, o, (const T*)qkv, ld,
                                        q_off, k_off, v_off, state, state_stride, seq_slots, H, D, V, ex)));
    return ti_check_launch("memory_token");
}
