// Long prompts through a matrix memory per (sequence, head) whose past fades by one number per token and head,
//
//   S_t = a_t S_(t-1) + b_t k_t v_t^T,   n_t = a_t n_(t-1) + b_t k_t,   o_t = S_t^T q_t
//
// (retention: a_t = the head's decay, b_t = 1, no n; the gated cell: a_t = keep, b_t = add; the state-space cell: a_t = e^(l_t), b_t = dt_t, no
// n, q and k shared by the heads of a group, and D_h v_t added to o_t). Instead of walking the tokens one by one, a
// sequence's tokens of the step are cut into chunks of 64, counted from the step's first. With L_t the sum of ln a up to t inside a chunk
// and S the state ahead of it,
//
//   o_t = e^(L_t) S^T q_t + sum_(s <= t) e^(L_t - L_s) b_s (q_t . k_s) v_s          n_t . q_t likewise with 1 for v_s
//   S  <- e^(L_64) S + sum_s e^(L_64 - L_s) b_s k_s v_s^T
//
// which is three products of matrices per chunk, all in 32-bit on the FMA units, and fills the device from one prompt:
//
//   memory_chunk_states   the sum in the second line, for every chunk at once
//   memory_chunk_scan     the states ahead of every chunk, element by element in chunk order; the sequence's state moves on
//   memory_chunk_outputs  the first line for every chunk at once, and where a block holds a head's whole row its divisor, RMS norm, weight
//                         and output gate as well
//
// q and k are rotated by the token's position and scaled while they are staged, in 32-bit. L is summed in 64-bit: a difference of two
// large sums must not lose the small decay between neighbours.
#include "chunk_index.cuh"
#include "mma_util.cuh"

#define MC_TOKENS CHUNK_TOKENS
#define MC_SLAB 128              // key rows and value columns staged at once
#define MC_PITCH (MC_SLAB + 4)   // floats between staged rows: eight rows' 16-byte pieces lie in different banks
#define MC_THREADS 256
#define MC_S_ROWS 16             // rows of the state staged at once, twice: one piece is on its way while the other is worked on
#define MC_FLOOR 1e-6f

struct ChunkArgs {
    const void* rows;            // [n, ld] of T: q at q_off (H * D), k at k_off, v at v_off (H * V), the output gate at g_off (H * V)
    long long ld;
    int q_off, k_off, v_off, g_off;
    const int* cu_seqlens;
    const int* positions;
    int B, H, D, V;
    const float* decay;          // [H], or null: coef [n, H, 2] = (keep, add)
    const float* coef;
    int coef_log;                // coef holds (ln keep, add)
    int vector;                  // there is a vector n beside S
    int per_qk;                  // heads that share a q and a k
    const float* skip;           // [H] or null: skip[h] * v joins o
    const float* cos_sin;        // [positions, rotary / 2, 2] or null
    int rotary;
    float q_scale, k_scale;
    float* ws;                   // [chunks, H, pitch]: S [D, V], then n [D]
    long long ws_pitch;
    float* total;                // [chunks, H]: e^(L_64)
};

// L and b of the chunk's tokens (beyond `count`: L stays, b is zero). 64 threads; the caller synchronises.
__device__ __forceinline__ void chunk_decays(const ChunkArgs& a, int h, int t0, int count, double* L, float* add) {
    if (threadIdx.x >= MC_TOKENS) return;
    const int s = threadIdx.x, lane = s & 31;
    double l = 0.0;
    float b = 0.f;
    if (s < count) {
        float log_keep = 0.f;
        b = 1.f;
        if (a.coef != nullptr) {
            const float2 c = __ldcg(reinterpret_cast<const float2*>(a.coef) + (size_t)(t0 + s) * a.H + h);
            log_keep = a.coef_log ? c.x : logf(c.x);
            b = c.y;
        } else {
            log_keep = logf(a.decay[h]);
        }
        l = (double)fmaxf(log_keep, -100.f);          // (e^-100 is zero beside anything 32-bit)
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double p = __shfl_up_sync(0xffffffffu, l, o);
        if (lane >= o) l += p;
    }
    L[s] = l;                                            // the second warp's share lacks the first's total: see chunk_join
    add[s] = b;
}
__device__ __forceinline__ void chunk_join(double* L) {
    const double first = L[31];
    __syncthreads();
    if (threadIdx.x >= 32 && threadIdx.x < MC_TOKENS) L[threadIdx.x] += first;
    __syncthreads();
}

// dst[token][0 .. MC_SLAB) (MC_PITCH apart) = the elements d0 .. of head h's q or k, rotated and scaled; zeros beyond the head and the chunk.
template <typename T, bool VECTORS>
__device__ __forceinline__ void stage_qk(const ChunkArgs& a, float* dst, int off, float scale, int h, int t0, int count, int d0) {
    const int D = a.D, half = a.rotary >> 1, width = min(MC_SLAB, (D - d0 + 3) / 4 * 4);
    if constexpr (VECTORS) {
        constexpr int VEC = Vec16<T>::N;
        const int per = width / VEC;
#pragma unroll 4
        for (int e = threadIdx.x; e < MC_TOKENS * per; e += MC_THREADS) {
            const int s = e / per, d = d0 + (e % per) * VEC;
            float* out = dst + s * MC_PITCH + d - d0;
            Vec16<T> v;
            if (s < count) {
                const T* row = (const T*)a.rows + (size_t)(t0 + s) * a.ld + off + (size_t)(h / a.per_qk) * D;
                v.load_cg(row + d);
                if (a.cos_sin != nullptr && d < a.rotary) {
                    const bool low = d < half;
                    Vec16<T> w;
                    w.load_cg(row + (low ? d + half : d - half));
                    const float4* cs = reinterpret_cast<const float4*>(a.cos_sin + ((size_t)__ldcg(a.positions + t0 + s) * half + (low ? d : d - half)) * 2);
                    const float sign = low ? -1.f : 1.f;
#pragma unroll
                    for (int i = 0; i < VEC; i += 2) {
                        const float4 c = __ldg(cs + i / 2);
                        v.v[i] = v.v[i] * c.x + sign * (w.v[i] * c.y);
                        v.v[i + 1] = v.v[i + 1] * c.z + sign * (w.v[i + 1] * c.w);
                    }
                }
#pragma unroll
                for (int i = 0; i < VEC; ++i) out[i] = v.v[i] * scale;
            } else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) out[i] = 0.f;
            }
        }
    } else {
        for (int e = threadIdx.x; e < MC_TOKENS * width; e += MC_THREADS) {
            const int s = e / width, d = d0 + e % width;
            float v = 0.f;
            if (s < count && d < D) {
                const T* row = (const T*)a.rows + (size_t)(t0 + s) * a.ld + off + (size_t)(h / a.per_qk) * D;
                v = to_f32(__ldcg(row + d));
                if (a.cos_sin != nullptr && d < a.rotary) {
                    const bool low = d < half;
                    const float2 c = __ldg(reinterpret_cast<const float2*>(a.cos_sin) + (size_t)__ldcg(a.positions + t0 + s) * half + (low ? d : d - half));
                    const float w = to_f32(__ldcg(row + (low ? d + half : d - half)));
                    v = v * c.x + (low ? -1.f : 1.f) * (w * c.y);
                }
                v *= scale;
            }
            dst[s * MC_PITCH + d - d0] = v;
        }
    }
}

// dst[token][0 .. MC_SLAB) = weight[token] times the columns v0 .. of head h's values; zeros beyond the head and the chunk.
template <typename T, bool VECTORS>
__device__ __forceinline__ void stage_v(const ChunkArgs& a, float* dst, const float* weight, int h, int t0, int count, int v0) {
    constexpr int VEC = VECTORS ? Vec16<T>::N : 1;
    const int per = MC_SLAB / VEC;
#pragma unroll 4
    for (int e = threadIdx.x; e < MC_TOKENS * per; e += MC_THREADS) {
        const int s = e / per, c = (e % per) * VEC;
        float* out = dst + s * MC_SLAB + c;
        const bool in = s < count && v0 + c < a.V;
        const T* src = (const T*)a.rows + (size_t)(t0 + s) * a.ld + a.v_off + (size_t)h * a.V + v0 + c;
        const float w = weight != nullptr ? weight[s] : 1.f;
        if constexpr (VECTORS) {
            Vec16<T> v;
            if (in) v.load_cg(src);
#pragma unroll
            for (int i = 0; i < VEC; ++i) out[i] = in ? v.v[i] * w : 0.f;
        } else {
            out[0] = in ? to_f32(__ldcg(src)) * w : 0.f;
        }
    }
}

// grid (chunks, H, slabs of keys x slabs of values). A thread owns 8 x 8 elements of the 128 x 128 block of the sum.
template <typename T, bool VECTORS>
__global__ void __launch_bounds__(MC_THREADS, 2) memory_chunk_states_kernel(ChunkArgs a) {
    extern __shared__ __align__(16) float smem[];
    float* ks = smem;                                    // [64][MC_PITCH]
    float* vs = ks + MC_TOKENS * MC_PITCH;               // [64][MC_SLAB], times the token's weight
    __shared__ double L[MC_TOKENS];
    __shared__ float add[MC_TOKENS], weight[MC_TOKENS];
    const int h = blockIdx.y, v_slabs = (a.V + MC_SLAB - 1) / MC_SLAB;
    const int d0 = (blockIdx.z / v_slabs) * MC_SLAB, v0 = (blockIdx.z % v_slabs) * MC_SLAB;
    int t0 = 0, count = 0;
    pdl_enter();
    if (!chunk_of(a.cu_seqlens, a.B, blockIdx.x, t0, count)) return;
    chunk_decays(a, h, t0, count, L, add);
    __syncthreads();
    chunk_join(L);
    if (threadIdx.x < MC_TOKENS) weight[threadIdx.x] = add[threadIdx.x] * expf((float)(L[MC_TOKENS - 1] - L[threadIdx.x]));
    if (blockIdx.z == 0 && threadIdx.x == 0) a.total[(size_t)blockIdx.x * a.H + h] = expf((float)L[MC_TOKENS - 1]);
    __syncthreads();
    stage_qk<T, VECTORS>(a, ks, a.k_off, a.k_scale, h, t0, count, d0);
    stage_v<T, VECTORS>(a, vs, weight, h, t0, count, v0);
    __syncthreads();
    const int cx = threadIdx.x & 15, ry = threadIdx.x >> 4;
    float acc[8][8];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
#pragma unroll 4
    for (int s = 0; s < MC_TOKENS; ++s) {
        const float4 k0 = *reinterpret_cast<const float4*>(ks + s * MC_PITCH + ry * 4), k1 = *reinterpret_cast<const float4*>(ks + s * MC_PITCH + 64 + ry * 4);
        const float4 v0_ = *reinterpret_cast<const float4*>(vs + s * MC_SLAB + cx * 4), v1_ = *reinterpret_cast<const float4*>(vs + s * MC_SLAB + 64 + cx * 4);
        const float kk[8] = {k0.x, k0.y, k0.z, k0.w, k1.x, k1.y, k1.z, k1.w}, vv[8] = {v0_.x, v0_.y, v0_.z, v0_.w, v1_.x, v1_.y, v1_.z, v1_.w};
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(kk[i], vv[j], acc[i][j]);
    }
    float* out = a.ws + ((size_t)blockIdx.x * a.H + h) * a.ws_pitch;
    const bool whole = a.V % 4 == 0;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = d0 + (i < 4 ? 0 : 64) + ry * 4 + (i & 3);
        if (d >= a.D) continue;
#pragma unroll
        for (int g = 0; g < 2; ++g) {
            const int v = v0 + g * 64 + cx * 4;
            if (whole && v < a.V) *reinterpret_cast<float4*>(out + (size_t)d * a.V + v) = make_float4(acc[i][4 * g], acc[i][4 * g + 1], acc[i][4 * g + 2], acc[i][4 * g + 3]);
            else
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (v + j < a.V) out[(size_t)d * a.V + v + j] = acc[i][4 * g + j];
        }
    }
    if (a.vector && v0 == 0 && threadIdx.x < MC_SLAB && d0 + threadIdx.x < a.D) {
        float n = 0.f;
        for (int s = 0; s < count; ++s) n = fmaf(weight[s], ks[s * MC_PITCH + threadIdx.x], n);
        out[(size_t)a.D * a.V + d0 + threadIdx.x] = n;
    }
}

// grid (elements, H, B): ws[chunk] becomes the state ahead of the chunk.
template <int VEC>
__global__ void __launch_bounds__(256) memory_chunk_scan_kernel(ChunkArgs a, float* state, long long state_stride, const int* seq_slots) {
    const int h = blockIdx.y, b = blockIdx.z;
    const int DV = a.D * a.V, elements = DV + (a.vector ? a.D : 0);
    const int e = (blockIdx.x * 256 + threadIdx.x) * VEC;
    pdl_enter();
    const int first = chunks_before(a.cu_seqlens, b);
    const int chunks = (__ldcg(a.cu_seqlens + b + 1) - __ldcg(a.cu_seqlens + b) + MC_TOKENS - 1) / MC_TOKENS;
    if (e >= elements) return;
    float* base = state + (size_t)__ldcg(seq_slots + b) * state_stride;
    float* st = e < DV ? base + (size_t)h * DV + e : base + (size_t)a.H * DV + (size_t)h * a.D + (e - DV);
    float* w = a.ws + ((size_t)first * a.H + h) * a.ws_pitch + e;
    const float* total = a.total + (size_t)first * a.H + h;
    const size_t step = (size_t)a.H * a.ws_pitch;
    float s[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) s[i] = __ldcg(st + i);
    constexpr int AHEAD = 8;
    for (int c = 0; c < chunks; c += AHEAD) {
        float m[AHEAD][VEC], f[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c + j >= chunks) break;
            f[j] = __ldcg(total + (size_t)(c + j) * a.H);
            if constexpr (VEC == 4) {
                const float4 t = __ldcg(reinterpret_cast<const float4*>(w + (size_t)(c + j) * step));
                m[j][0] = t.x; m[j][1] = t.y; m[j][2] = t.z; m[j][3] = t.w;
            } else {
                m[j][0] = __ldcg(w + (size_t)(c + j) * step);
            }
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c + j >= chunks) break;
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(w + (size_t)(c + j) * step) = make_float4(s[0], s[1], s[2], s[3]);
            else w[(size_t)(c + j) * step] = s[0];
#pragma unroll
            for (int i = 0; i < VEC; ++i) s[i] = fmaf(f[j], s[i], m[j][i]);
        }
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) st[i] = s[i];
}

struct ChunkOut {
    void* y;                     // [n, H * V] of T: the normed and gated heads (V <= MC_SLAB), or null
    float* o;                    // [n, H * V]: the raw heads
    float* nq;                   // [n, H] (raw heads of the gated cell)
    const float* em;             // [n, H] = e^(-m) (gated cell)
    const void* w;               // [H * V] of T or null
    int gate_sigmoid;
    float eps;
};

// grid (chunks, H, slabs of values). A thread owns rows 4 ry .. 4 ry + 3 and columns 4 cx .. and 64 + 4 cx .. of the chunk's outputs.
template <typename T, bool VECTORS>
__global__ void __launch_bounds__(MC_THREADS, 2) memory_chunk_outputs_kernel(ChunkArgs a, ChunkOut out) {
    extern __shared__ __align__(16) float smem[];
    float* qs = smem;                                    // [64][MC_PITCH]
    float* ks = qs + MC_TOKENS * MC_PITCH;               // [64][MC_PITCH]; later P [64][68] and two pieces of the state [MC_S_ROWS][MC_SLAB]
    float* vs = ks + MC_TOKENS * MC_PITCH;               // [64][MC_SLAB]
    float* P = ks;
    float* ss = ks + MC_TOKENS * (MC_TOKENS + 4);
    __shared__ double L[MC_TOKENS];
    __shared__ float add[MC_TOKENS], past[MC_TOKENS], den[MC_TOKENS];
    const int h = blockIdx.y, v0 = blockIdx.z * MC_SLAB, D = a.D, V = a.V;
    const bool gated = a.vector != 0;
    int t0 = 0, count = 0;
    pdl_enter();
    if (!chunk_of(a.cu_seqlens, a.B, blockIdx.x, t0, count)) return;
    chunk_decays(a, h, t0, count, L, add);
    __syncthreads();
    chunk_join(L);
    if (threadIdx.x < MC_TOKENS) past[threadIdx.x] = expf((float)L[threadIdx.x]);
    const int cx = threadIdx.x & 15, ry = threadIdx.x >> 4;
    const float* state = a.ws + ((size_t)blockIdx.x * a.H + h) * a.ws_pitch;
    const float* n_prev = state + (size_t)D * V;
    // q . k of every pair of the chunk: rows 4 ry .., columns cx, cx + 16, ..
    float p[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) p[i][j] = 0.f;
    float qn = 0.f;                                      // this thread's share of q . n for row threadIdx.x / 4
    for (int d0 = 0; d0 < D; d0 += MC_SLAB) {
        if (d0 > 0) __syncthreads();
        stage_qk<T, VECTORS>(a, qs, a.q_off, a.q_scale, h, t0, count, d0);
        stage_qk<T, VECTORS>(a, ks, a.k_off, a.k_scale, h, t0, count, d0);
        if (d0 == 0) stage_v<T, VECTORS>(a, vs, nullptr, h, t0, count, v0);
        __syncthreads();
        const int width = min(MC_SLAB, (D - d0 + 3) / 4 * 4);
#pragma unroll 4
        for (int d = 0; d < width; d += 4) {
            float4 q4[4], k4[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) q4[i] = *reinterpret_cast<const float4*>(qs + (ry * 4 + i) * MC_PITCH + d);
#pragma unroll
            for (int j = 0; j < 4; ++j) k4[j] = *reinterpret_cast<const float4*>(ks + (cx + 16 * j) * MC_PITCH + d);
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    p[i][j] = fmaf(q4[i].x, k4[j].x, p[i][j]);
                    p[i][j] = fmaf(q4[i].y, k4[j].y, p[i][j]);
                    p[i][j] = fmaf(q4[i].z, k4[j].z, p[i][j]);
                    p[i][j] = fmaf(q4[i].w, k4[j].w, p[i][j]);
                }
        }
        if (gated) {
            const float* q = qs + (threadIdx.x >> 2) * MC_PITCH;
            for (int d = threadIdx.x & 3; d0 + d < D && d < MC_SLAB; d += 4) qn = fmaf(q[d], __ldcg(n_prev + d0 + d), qn);
        }
    }
    __syncthreads();                                     // the staged keys are done with: P and the state's pieces take their place
    const int pieces = (D + MC_S_ROWS - 1) / MC_S_ROWS;
    auto fetch = [&](int piece) {                        // rows piece * MC_S_ROWS .. of the state, zeros beyond
        float* dst = ss + (piece & 1) * MC_S_ROWS * MC_SLAB;
        const int d = piece * MC_S_ROWS;
        if (V % 4 == 0) {
            for (int e = threadIdx.x; e < MC_S_ROWS * (MC_SLAB / 4); e += MC_THREADS) {
                const int r = e / (MC_SLAB / 4), c = (e % (MC_SLAB / 4)) * 4;
                if (d + r < D && v0 + c < V) cp_async16(smem_u32(dst + r * MC_SLAB + c), state + (size_t)(d + r) * V + v0 + c);
                else *reinterpret_cast<float4*>(dst + r * MC_SLAB + c) = make_float4(0.f, 0.f, 0.f, 0.f);
            }
        } else {
            for (int e = threadIdx.x; e < MC_S_ROWS * MC_SLAB; e += MC_THREADS) {
                const int r = e / MC_SLAB, c = e % MC_SLAB;
                dst[e] = d + r < D && v0 + c < V ? __ldcg(state + (size_t)(d + r) * V + v0 + c) : 0.f;
            }
        }
        cp_async_commit();
    };
    fetch(0);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = ry * 4 + i, s = cx + 16 * j;
            P[t * (MC_TOKENS + 4) + s] = s <= t ? p[i][j] * (add[s] * expf((float)(L[t] - L[s]))) : 0.f;
        }
    // The past's share: q S, a piece of the state's rows at a time.
    float acc[4][8];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
    for (int piece = 0; piece < pieces; ++piece) {
        const int d = piece * MC_S_ROWS, in_slab = d % MC_SLAB;
        cp_async_wait<0>();
        __syncthreads();                                 // this piece is there, and everyone is done with the one before
        if (piece + 1 < pieces) fetch(piece + 1);
        if (D > MC_SLAB && in_slab == 0) {               // (with one slab q is still staged)
            stage_qk<T, VECTORS>(a, qs, a.q_off, a.q_scale, h, t0, count, d);
            __syncthreads();
        }
        const float* sp = ss + (piece & 1) * MC_S_ROWS * MC_SLAB;
        const int padded = min(MC_S_ROWS, (D - d + 3) / 4 * 4);          // (the staged q is zero beyond the head)
#pragma unroll 2
        for (int r = 0; r < padded; r += 4) {
            float4 q4[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) q4[i] = *reinterpret_cast<const float4*>(qs + (ry * 4 + i) * MC_PITCH + in_slab + r);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float4 s0 = *reinterpret_cast<const float4*>(sp + (r + k) * MC_SLAB + cx * 4), s1 = *reinterpret_cast<const float4*>(sp + (r + k) * MC_SLAB + 64 + cx * 4);
                const float sv[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float q = k == 0 ? q4[i].x : k == 1 ? q4[i].y : k == 2 ? q4[i].z : q4[i].w;
#pragma unroll
                    for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(q, sv[j], acc[i][j]);
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float w = past[ry * 4 + i];
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] *= w;
    }
    // The chunk's own share: P v. (P was written before the barriers above; a head of no rows does not exist.)
    const int last = min(MC_TOKENS, ry * 4 + 4);         // later tokens' weights are zero
    for (int s = 0; s < last; s += 4) {
        float4 p4[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) p4[i] = *reinterpret_cast<const float4*>(P + (ry * 4 + i) * (MC_TOKENS + 4) + s);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float4 s0 = *reinterpret_cast<const float4*>(vs + (s + k) * MC_SLAB + cx * 4), s1 = *reinterpret_cast<const float4*>(vs + (s + k) * MC_SLAB + 64 + cx * 4);
            const float sv[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float w = k == 0 ? p4[i].x : k == 1 ? p4[i].y : k == 2 ? p4[i].z : p4[i].w;
#pragma unroll
                for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(w, sv[j], acc[i][j]);
            }
        }
    }
    if (gated) {                                         // n . q of every row: four threads a row
        const int t = threadIdx.x >> 2, part = threadIdx.x & 3;
        float own = 0.f;
        for (int s = part; s <= t; s += 4) own += P[t * (MC_TOKENS + 4) + s];
        float nq = fmaf(past[t], qn, own);
        nq += __shfl_xor_sync(0xffffffffu, nq, 1);
        nq += __shfl_xor_sync(0xffffffffu, nq, 2);
        if (part == 0 && t < count) {
            if (out.y != nullptr) den[t] = 1.0f / (fmaxf(fabsf(nq), __ldcg(out.em + (size_t)(t0 + t) * a.H + h)) + MC_FLOOR);
            else if (blockIdx.z == 0) out.nq[(size_t)(t0 + t) * a.H + h] = nq;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ry * 4 + i;
        const bool in = t < count;
        const size_t at = (size_t)(t0 + t) * a.H * V + (size_t)h * V + v0;
        if (out.y == nullptr) {
            if (in)
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const int c = (j < 4 ? 0 : 64) + cx * 4 + (j & 3);
                    if (v0 + c < V) out.o[at + c] = a.skip != nullptr ? fmaf(a.skip[h], vs[t * MC_SLAB + c], acc[i][j]) : acc[i][j];
                }
            continue;
        }
        float square = 0.f;
        const float d = gated && in ? den[t] : 1.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {                    // (columns beyond the head are zero)
            acc[i][j] *= d;
            square = fmaf(acc[i][j], acc[i][j], square);
        }
#pragma unroll
        for (int m = 1; m < 16; m <<= 1) square += __shfl_xor_sync(0xffffffffu, square, m);
        const float inv = 1.0f / sqrtf(square / (float)V + out.eps);
        if (!in) continue;
        const T* gate = (const T*)a.rows + (size_t)(t0 + t) * a.ld + a.g_off + (size_t)h * V;
        const T* w = (const T*)out.w;
        T* y = (T*)out.y + at;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = (j < 4 ? 0 : 64) + cx * 4 + (j & 3);
            if (c < V) {
                const float g = to_f32(__ldcg(gate + c));
                float v = acc[i][j] * inv;
                if (w != nullptr) v *= to_f32(w[(size_t)h * V + c]);
                y[c] = from_f32<T>(v * ((out.gate_sigmoid ? 1.0f : g) / (1.0f + expf(-g))));
            }
        }
    }
}

static int launch_chunks(const ChunkArgs& a, const ChunkOut& out, float* state, long long state_stride, int chunks, const int* seq_slots, int dtype,
                         cudaStream_t stream) {
    const int d_slabs = (a.D + MC_SLAB - 1) / MC_SLAB, v_slabs = (a.V + MC_SLAB - 1) / MC_SLAB;
    const size_t smem_s = (size_t)MC_TOKENS * (MC_PITCH + MC_SLAB) * sizeof(float), smem_o = (size_t)MC_TOKENS * (2 * MC_PITCH + MC_SLAB) * sizeof(float);
    const bool scan4 = a.D % 4 == 0 && (a.D * a.V) % 4 == 0 && state_stride % 4 == 0 && aligned16(state) && aligned16(a.ws);
    const int elements = a.D * a.V + (a.vector ? a.D : 0);
    TI_DISPATCH_DTYPE(dtype, {
        constexpr int VEC = Vec16<T>::N;
        const bool vectors = aligned16(a.rows) && a.ld % VEC == 0 && a.q_off % VEC == 0 && a.k_off % VEC == 0 && a.v_off % VEC == 0 && a.D % VEC == 0 && a.V % VEC == 0 &&
                             (a.cos_sin == nullptr || ((a.rotary / 2) % VEC == 0 && aligned16(a.cos_sin)));
        static bool configured = false;                  // per element type
        if (!configured) {
            cudaError_t e = cudaFuncSetAttribute(memory_chunk_states_kernel<T, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_s);
            if (e == cudaSuccess) e = cudaFuncSetAttribute(memory_chunk_states_kernel<T, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_s);
            if (e == cudaSuccess) e = cudaFuncSetAttribute(memory_chunk_outputs_kernel<T, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_o);
            if (e == cudaSuccess) e = cudaFuncSetAttribute(memory_chunk_outputs_kernel<T, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_o);
            if (e != cudaSuccess) return ti_fail("memory_chunks: %s", cudaGetErrorString(e));
            configured = true;
        }
        const dim3 grid_s(chunks, a.H, d_slabs * v_slabs), grid_o(chunks, a.H, v_slabs);
        if (vectors) ti_launch(memory_chunk_states_kernel<T, true>, grid_s, dim3(MC_THREADS), smem_s, stream, a);
        else ti_launch(memory_chunk_states_kernel<T, false>, grid_s, dim3(MC_THREADS), smem_s, stream, a);
        if (int rc = ti_check_launch("memory_chunk_states")) return rc;
        if (scan4) ti_launch(memory_chunk_scan_kernel<4>, dim3((elements / 4 + 255) / 256, a.H, a.B), dim3(256), 0, stream, a, state, state_stride, seq_slots);
        else ti_launch(memory_chunk_scan_kernel<1>, dim3((elements + 255) / 256, a.H, a.B), dim3(256), 0, stream, a, state, state_stride, seq_slots);
        if (int rc = ti_check_launch("memory_chunk_scan")) return rc;
        if (vectors) ti_launch(memory_chunk_outputs_kernel<T, true>, grid_o, dim3(MC_THREADS), smem_o, stream, a, out);
        else ti_launch(memory_chunk_outputs_kernel<T, false>, grid_o, dim3(MC_THREADS), smem_o, stream, a, out);
    });
    return ti_check_launch("memory_chunk_outputs");
}

// Floats of work space per (chunk, head).
extern "C" int ti_memory_chunk_pitch(int D, int V) { return (D * V + D + 3) / 4 * 4; }

// `chunks` = sum over the sequences of ceil(tokens / 64); ws [chunks, H, ti_memory_chunk_pitch] and total [chunks, H] float are work space.
// decay [H] (retention) or coef [n, H, 2] and em [n, H] (the gated cell). y [n, H * V] for heads of up to 128 values, else o (and nq).
extern "C" int ti_memory_chunks(void* y, float* o, float* nq, const float* em, const void* rows, long long ld, int q_off, int k_off, int v_off, int g_off,
                                float* state, long long state_stride, const float* decay, const float* coef, const float* cos_sin, int rotary,
                                const int* positions, float q_scale, float k_scale, const void* w, int gate_sigmoid, float eps, float* ws, float* total,
                                int chunks, const int* cu_seqlens, const int* seq_slots, int B, int H, int D, int V, int dtype, cudaStream_t stream) {
    if (B == 0 || chunks == 0) return 0;
    TI_REQUIRE((decay != nullptr) != (coef != nullptr) && (y != nullptr) != (o != nullptr), "memory_chunks: one decay per head or coefficients, y or o");
    TI_REQUIRE(y == nullptr || V <= MC_SLAB, "memory_chunks: a head of %d values is shared out between blocks", V);
    TI_REQUIRE(coef == nullptr || (y != nullptr ? em != nullptr : nq != nullptr), "memory_chunks: the gated cell needs its divisor's pieces");
    TI_REQUIRE(H > 0 && D > 0 && V > 0 && H <= 65535 && B <= 65535, "memory_chunks: %d heads of %d x %d, %d sequences", H, D, V, B);
    TI_REQUIRE(cos_sin == nullptr || (positions != nullptr && rotary >= 2 && rotary % 2 == 0 && rotary <= D), "memory_chunks: rotation over %d of %d", rotary, D);
    const ChunkArgs a = {rows, ld, q_off, k_off, v_off, g_off, cu_seqlens, positions, B, H, D, V, decay, coef, 0, coef != nullptr, 1, nullptr, cos_sin,
                         cos_sin != nullptr ? rotary : 0, q_scale, k_scale, ws, ti_memory_chunk_pitch(D, V), total};
    const ChunkOut out = {y, o, nq, em, w, gate_sigmoid, eps};
    return launch_chunks(a, out, state, state_stride, chunks, seq_slots, dtype, stream);
}

// The state-space cell: rows [n, ld] of T with x (H * V columns) at x_off, B and C (groups * N each) at b_off and c_off; coef [n, H, 2] = (l, dt);
// o [n, H * V] float = y with the skip in it. Work space as above.
extern "C" int ti_ssm_chunks(float* o, const void* rows, long long ld, int x_off, int b_off, int c_off, float* state, long long state_stride,
                             const float* coef, const float* skip, float* ws, float* total, int chunks, const int* cu_seqlens, const int* seq_slots,
                             int B, int H, int groups, int N, int V, int dtype, cudaStream_t stream) {
    if (B == 0 || chunks == 0) return 0;
    TI_REQUIRE(H > 0 && groups > 0 && H % groups == 0 && N > 0 && V > 0 && H <= 65535 && B <= 65535, "ssm_chunks: %d heads in %d groups, %d x %d", H, groups, N, V);
    const ChunkArgs a = {rows, ld, c_off, b_off, x_off, 0, cu_seqlens, nullptr, B, H, N, V, nullptr, coef, 1, 0, H / groups, skip, nullptr, 0, 1.f, 1.f, ws,
                         ti_memory_chunk_pitch(N, V), total};
    const ChunkOut out = {nullptr, o, nullptr, nullptr, nullptr, 0, 0.f};
    return launch_chunks(a, out, state, state_stride, chunks, seq_slots, dtype, stream);
}
