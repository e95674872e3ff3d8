// Linear attention with a decay per head ("lightning" attention): a matrix state per (sequence, head) that is carried
// from token to token,
//
//   S_t = a_h S_(t-1) + k_t v_t^T        S [dim, vdim], 32-bit, zero at the start of a sequence
//   o_t = S_t^T q_t                      [vdim]
//
// with q, k, v = act(projection) (act: SiLU or none; the activation is applied, and rounded to T, as the rows are read).
//
//   lightning_scan   the recurrence over the tokens a step brings, from the state the earlier steps left; the new state is
//                    written back. One kernel serves prompts and one-token steps.
//   lightning_out    y = T( o / rms(o) * w * sigmoid(g) ): the RMS norm over all heads' outputs together, in 32-bit, times
//                    the output gate; the input of the output projection.
//
// The scan: the columns of S are independent (column j of S sees v_t[j] only), so a block owns 32 columns of one
// (sequence, head) and walks the sequence's tokens in order; its 8 or 16 warps split the rows of S (warp w owns DP rows in a
// row, read from shared memory four at a time), a lane owns one column, the state lives in registers. Tokens are staged 32 at a time in shared memory; the
// warps' partial sums of o meet there once per 32 tokens. A launch of few blocks (one prompt, few heads) shares the rows of S
// out between two blocks per column block, whose two shares of o are added in global memory. A token's result depends on
// the sequence's earlier tokens alone; the order of its sums depends on the sizes and on whether the launch was shared
// out, so results agree to rounding, not bit for bit, between a prompt alone and the same prompt in a large batch.
// Everything is 32-bit arithmetic; nothing of the state, the decay or o is rounded.
#include "lightning_scan.cuh"

// One token per sequence: the step reads and writes every state once and is bound by that traffic. A block owns 128 columns
// of one (sequence, head): a lane owns four of them (16 bytes of a row), the warps take the rows in turn with several rows'
// loads in flight, and their shares of o meet in shared memory. The arithmetic per element is the scan's.
#define LT_WARPS 8
template <typename T>
__global__ void __launch_bounds__(LT_WARPS * 32) lightning_token_kernel(float* __restrict__ o, const T* qkv, long long ld, int q_off, int k_off,
                                                                        int v_off, float* state, const float* __restrict__ decay,
                                                                        const int* seq_slots, int H, int D, int V, int act) {
    extern __shared__ float smem[];
    float* qs = smem;                                   // [D]
    float* ks = qs + D;                                 // [D]
    float* part = ks + D;                               // [LT_WARPS][128]
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
    const int col = blockIdx.x * 128 + lane * 4, h = blockIdx.y, b = blockIdx.z;
    const float a = decay[h];
    pdl_enter();
    const T* row = qkv + (size_t)b * ld;
    for (int d = threadIdx.x; d < D; d += LT_WARPS * 32) {
        float qv = to_f32(__ldcg(row + q_off + (size_t)h * D + d)), kv = to_f32(__ldcg(row + k_off + (size_t)h * D + d));
        if (act) { qv = rnd<T>(silu_value(qv)); kv = rnd<T>(silu_value(kv)); }
        qs[d] = qv;
        ks[d] = kv;
    }
    float v4[4] = {0.f, 0.f, 0.f, 0.f};
    if (col < V) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            v4[e] = to_f32(__ldcg(row + v_off + (size_t)h * V + col + e));
            if (act) v4[e] = rnd<T>(silu_value(v4[e]));
        }
    }
    __syncthreads();
    float* S = state + ((size_t)__ldcg(seq_slots + b) * H + h) * D * V;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (col < V) {
#pragma unroll 4
        for (int d = w; d < D; d += LT_WARPS) {
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
    __syncthreads();
    for (int c = threadIdx.x; c < 128; c += LT_WARPS * 32) {
        if (blockIdx.x * 128 + c >= V) continue;
        float sum = 0.f;
#pragma unroll
        for (int p = 0; p < LT_WARPS; ++p) sum += part[p * 128 + c];
        o[(size_t)b * H * V + (size_t)h * V + blockIdx.x * 128 + c] = sum;
    }
}

// o [n, H * V] float; qkv [n, ld] of T with the heads' queries from column q_off on (H * D of them), keys from k_off, values
// from v_off (H * V); state [slots, H, D, V] float; decay [H] float; cu_seqlens [B + 1], seq_slots [B] (n_tokens in all). act: 1 = SiLU.
extern "C" int ti_lightning_scan(float* o, const void* qkv, long long ld, int q_off, int k_off, int v_off, float* state, const float* decay,
                                 const int* cu_seqlens, const int* seq_slots, int n_tokens, int B, int H, int D, int V, int act, int dtype,
                                 cudaStream_t stream) {
    if (B == 0) return 0;
    TI_REQUIRE(H > 0 && D > 0 && V > 0 && D <= LS_MAX_DIM, "lightning_scan: %d heads of %d x %d (the key size is at most %d)", H, D, V, LS_MAX_DIM);
    TI_REQUIRE(H <= 65535 && B <= 65535, "lightning_scan: %d heads, %d sequences", H, B);
    if (n_tokens == B && V % 4 == 0 && D <= 2048) {      // one token per sequence: the kernel that streams the states
        const size_t smem1 = (size_t)(2 * D + LT_WARPS * 128) * sizeof(float);
        TI_DISPATCH_DTYPE(dtype, (ti_launch(lightning_token_kernel<T>, dim3((V + 127) / 128, H, B), dim3(LT_WARPS * 32), smem1, stream, o, (const T*)qkv, ld,
                                            q_off, k_off, v_off, state, decay, seq_slots, H, D, V, act)));
        return ti_check_launch("lightning_scan");
    }
    ScanExtras ex = {};
    ex.state_stride = (long long)H * D * V;
    ex.q_scale = ex.k_scale = 1.f;
    return launch_lightning_scan<0>("lightning_scan", o, qkv, ld, q_off, k_off, v_off, state, decay, cu_seqlens, seq_slots, n_tokens, B, H, D, V, act, ex,
                                    dtype, stream);
}

template <typename T>
__global__ void lightning_out_kernel(T* __restrict__ y, const float* o, const T* g, long long ldg, const T* __restrict__ w, float eps, int size) {
    __shared__ float scratch[33];
    const float* row = o + (size_t)blockIdx.x * size;
    float ss = 0.f;
    pdl_enter();
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        const float v = __ldcg(row + i);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)size + eps);
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
        float v = __ldcg(row + i) * inv * to_f32(w[i]);
        if (g != nullptr) v = v / (1.0f + expf(-to_f32(__ldcg(g + (size_t)blockIdx.x * ldg + i))));
        y[(size_t)blockIdx.x * size + i] = from_f32<T>(v);
    }
}

// y [n, size] = T(o / rms(o) * w * sigmoid(g)); o [n, size] float, g [n, ldg] of T (null: no gate), w [size].
extern "C" int ti_lightning_out(void* y, const float* o, const void* g, long long ldg, const void* w, float eps, int n, int size, int dtype,
                                cudaStream_t stream) {
    if (n == 0) return 0;
    TI_REQUIRE(size > 0, "lightning_out: size %d", size);
    const int threads = size >= 4096 ? 512 : size >= 1024 ? 256 : 128;
    TI_DISPATCH_DTYPE(dtype, (ti_launch(lightning_out_kernel<T>, dim3(n), dim3(threads), 0, stream, (T*)y, o, (const T*)g, ldg, (const T*)w, eps, size)));
    return ti_check_launch("lightning_out");
}
