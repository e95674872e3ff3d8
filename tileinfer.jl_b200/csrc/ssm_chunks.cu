// The chunked form of the state-space recurrence (memory_chunks.cu has the equations and the 32-bit form) with its products on the tensor
// cores, for bfloat16 rows. x, B and C are bfloat16 as they come; what is 32-bit (the weights dt e^(L - L_s), the weighted scores and the
// state) enters a product as a sum of two bfloat16 numbers, hi + lo, whose error is 2^-17 of its value, with 32-bit accumulation:
//
//   ssm_chunk_states    sum_s B_s (w_s x_s)^T of every chunk, w_s = dt_s e^(L_end - L_s): B^T [state x 64] times (hi + lo) [64 x vdim]
//   ssm_chunk_scan      the states ahead of every chunk, in 32-bit element by element; they are left as hi and lo, eight elements of each in turn
//   ssm_chunk_outputs   y = e^L (C S) + P x + D x, P = (C B^T) . (dt_s e^(L_t - L_s)) for s <= t
//
// A block takes one chunk of up to four heads of a group, which share B, C and C B^T. Sums of ln decays are kept as two floats in base 2.
#include "chunk_index.cuh"
#include "mma_util.cuh"

#define SC_THREADS 128
#define SC_VALUES 64                     // value columns of a block
#define SC_ROWS 128                      // state rows of a block of ssm_chunk_states
#define SC_X_PITCH (SC_VALUES + 8)       // bfloat16 elements between staged rows: an odd number of 16-byte pieces, so ldmatrix is free of conflicts
#define SC_S_PITCH (2 * SC_VALUES + 8)
#define SC_MAX_HEADS 4

struct SsmChunkArgs {
    const bf16* rows;
    long long ld;
    int x_off, b_off, c_off;
    const float* coef;                   // [n, H, 2] = (l, dt)
    const float* skip;                   // [H]
    const int* cu_seqlens;
    int B, H, per_group, heads, N, V;    // heads: how many a block takes
    float* ws;
    long long ws_pitch;
    float* total;
    float* y;
};

struct Decays {                          // of one head's 64 tokens: L (base 2, hi + lo), dt
    float hi[CHUNK_TOKENS], lo[CHUNK_TOKENS], dt[CHUNK_TOKENS];
};

// The sums of the block's heads: a warp takes a head's tokens 32 at a time. The caller synchronises.
__device__ __forceinline__ void load_decays(const SsmChunkArgs& a, Decays* out, int h0, int t0, int count) {
    const int lane = threadIdx.x & 31;
    for (int i = threadIdx.x >> 5; i < a.heads; i += SC_THREADS / 32) {
        double before = 0.0;
#pragma unroll
        for (int part = 0; part < CHUNK_TOKENS / 32; ++part) {
            const int s = part * 32 + lane;
            float2 c = make_float2(0.f, 0.f);
            if (s < count) c = __ldcg(reinterpret_cast<const float2*>(a.coef) + (size_t)(t0 + s) * a.H + h0 + i);
            double l = (double)fmaxf(c.x, -100.f) * 1.4426950408889634;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double p = __shfl_up_sync(0xffffffffu, l, o);
                if (lane >= o) l += p;
            }
            l += before;
            const float hi = (float)l;
            out[i].hi[s] = hi;
            out[i].lo[s] = (float)(l - (double)hi);
            out[i].dt[s] = c.y;
            before = __shfl_sync(0xffffffffu, l, 31);
        }
    }
}
// e^(L_t - L_s)
__device__ __forceinline__ float decay_between(const Decays& d, int t, int s) { return exp2f((d.hi[t] - d.hi[s]) + (d.lo[t] - d.lo[s])); }

// v as hi + lo
__device__ __forceinline__ void split_pair(float v0, float v1, unsigned& hi, unsigned& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
    hi = *reinterpret_cast<const unsigned*>(&h);
    lo = pack_bf16(v0 - __low2float(h), v1 - __high2float(h));
}

// dst[token][0 .. width) of 16-byte pieces from column `col` of the step's rows, zeros beyond the chunk and beyond `valid` columns.
__device__ __forceinline__ void stage_rows(const SsmChunkArgs& a, bf16* dst, int pitch, int col, int width, int valid, int t0, int count) {
    const int per = width / 8;
    for (int e = threadIdx.x; e < CHUNK_TOKENS * per; e += SC_THREADS) {
        const int s = e / per, c = (e % per) * 8;
        bf16* to = dst + s * pitch + c;
        if (s < count && c < valid) cp_async16(smem_u32(to), a.rows + (size_t)(t0 + s) * a.ld + col + c);
        else *reinterpret_cast<uint4*>(to) = make_uint4(0u, 0u, 0u, 0u);
    }
}

// grid (chunks, H / heads, state slabs x value slabs). A warp owns 32 state rows.
__global__ void __launch_bounds__(SC_THREADS) ssm_chunk_states_kernel(SsmChunkArgs a) {
    extern __shared__ __align__(128) unsigned char smem_raw[];
    const int v_slabs = (a.V + SC_VALUES - 1) / SC_VALUES, n0 = (blockIdx.z / v_slabs) * SC_ROWS, v0 = (blockIdx.z % v_slabs) * SC_VALUES;
    const int rows = min(SC_ROWS, (a.N - n0 + 15) / 16 * 16), pitch = rows + 8, h0 = blockIdx.y * a.heads;
    bf16* bt = reinterpret_cast<bf16*>(smem_raw);        // [64][pitch]
    bf16* xh = bt + CHUNK_TOKENS * pitch;                // [64][SC_X_PITCH]
    bf16* xl = xh + CHUNK_TOKENS * SC_X_PITCH;
    __shared__ Decays dec[SC_MAX_HEADS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mat = lane >> 3, r = lane & 7, g = lane >> 2, t = lane & 3;
    int t0 = 0, count = 0;
    pdl_enter();
    if (!chunk_of(a.cu_seqlens, a.B, blockIdx.x, t0, count)) return;
    stage_rows(a, bt, pitch, a.b_off + (h0 / a.per_group) * a.N + n0, rows, a.N - n0, t0, count);
    cp_async_commit();
    constexpr int PIECES = CHUNK_TOKENS * (SC_VALUES / 8) / SC_THREADS;          // 16-byte pieces of x a thread stages per head
    uint4 raw[PIECES];
    auto fetch = [&](int h) {
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
            const int e = threadIdx.x + p * SC_THREADS, s = e / (SC_VALUES / 8), c = (e % (SC_VALUES / 8)) * 8;
            raw[p] = make_uint4(0u, 0u, 0u, 0u);
            if (s < count && v0 + c < a.V) raw[p] = __ldcg(reinterpret_cast<const uint4*>(a.rows + (size_t)(t0 + s) * a.ld + a.x_off + (size_t)h * a.V + v0 + c));
        }
    };
    fetch(h0);
    load_decays(a, dec, h0, t0, count);
    cp_async_wait<0>();
    __syncthreads();
    if (blockIdx.z == 0 && threadIdx.x < a.heads)
        a.total[(size_t)blockIdx.x * a.H + h0 + threadIdx.x] = exp2f(dec[threadIdx.x].hi[CHUNK_TOKENS - 1] + dec[threadIdx.x].lo[CHUNK_TOKENS - 1]);
    for (int i = 0; i < a.heads; ++i) {
        const Decays& d = dec[i];
        if (i > 0) __syncthreads();                      // the last head's x is done with
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
            const int e = threadIdx.x + p * SC_THREADS, s = e / (SC_VALUES / 8), c = (e % (SC_VALUES / 8)) * 8;
            const float w = d.dt[s] * decay_between(d, CHUNK_TOKENS - 1, s);
            Vec16<bf16> v;
            v.unpack(raw[p]);
            uint4 hi, lo;
            split_pair(v.v[0] * w, v.v[1] * w, hi.x, lo.x);
            split_pair(v.v[2] * w, v.v[3] * w, hi.y, lo.y);
            split_pair(v.v[4] * w, v.v[5] * w, hi.z, lo.z);
            split_pair(v.v[6] * w, v.v[7] * w, hi.w, lo.w);
            *reinterpret_cast<uint4*>(xh + s * SC_X_PITCH + c) = hi;
            *reinterpret_cast<uint4*>(xl + s * SC_X_PITCH + c) = lo;
        }
        if (i + 1 < a.heads) fetch(h0 + i + 1);
        __syncthreads();
        float acc[2][8][4];
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int c = 0; c < 8; ++c)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[m][c][e] = 0.f;
        if (warp * 32 < rows) {
#pragma unroll
            for (int kk = 0; kk < CHUNK_TOKENS / 16; ++kk) {
                unsigned af[2][4];
#pragma unroll
                for (int m = 0; m < 2; ++m)
                    if (warp * 32 + m * 16 < rows)
                        ldmatrix_x4_trans(af[m], smem_u32(bt + (kk * 16 + (mat >> 1) * 8 + r) * pitch + warp * 32 + m * 16 + (mat & 1) * 8));
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    const bf16* x = part ? xl : xh;
#pragma unroll
                    for (int c = 0; c < 8; c += 2) {
                        unsigned vb[4];
                        ldmatrix_x4_trans(vb, smem_u32(x + (kk * 16 + (mat & 1) * 8 + r) * SC_X_PITCH + (c + (mat >> 1)) * 8));
#pragma unroll
                        for (int m = 0; m < 2; ++m)
                            if (warp * 32 + m * 16 < rows) {
                                mma16816(acc[m][c], af[m], vb[0], vb[1]);
                                mma16816(acc[m][c + 1], af[m], vb[2], vb[3]);
                            }
                    }
                }
            }
            float* out = a.ws + ((size_t)blockIdx.x * a.H + h0 + i) * a.ws_pitch;
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int n = n0 + warp * 32 + m * 16 + half * 8 + g;
                    if (warp * 32 + m * 16 >= rows || n >= a.N) continue;
#pragma unroll
                    for (int c = 0; c < 8; ++c)
                        if (v0 + c * 8 < a.V) *reinterpret_cast<float2*>(out + (size_t)n * a.V + v0 + c * 8 + 2 * t) = make_float2(acc[m][c][2 * half], acc[m][c][2 * half + 1]);
                }
        }
    }
}

// grid (elements / 8, H, B): ws[chunk] becomes the state ahead of the chunk, eight elements' hi then their lo; the sequence's state moves on.
__global__ void __launch_bounds__(128) ssm_chunk_scan_kernel(SsmChunkArgs a, float* state, long long state_stride, const int* seq_slots) {
    const int h = blockIdx.y, b = blockIdx.z, elements = a.N * a.V, e = (blockIdx.x * 128 + threadIdx.x) * 8;
    pdl_enter();
    const int first = chunks_before(a.cu_seqlens, b);
    const int chunks = (__ldcg(a.cu_seqlens + b + 1) - __ldcg(a.cu_seqlens + b) + CHUNK_TOKENS - 1) / CHUNK_TOKENS;
    if (e >= elements) return;
    float4* st = reinterpret_cast<float4*>(state + (size_t)__ldcg(seq_slots + b) * state_stride + (size_t)h * elements + e);
    float* w = a.ws + ((size_t)first * a.H + h) * a.ws_pitch + e;
    const float* total = a.total + (size_t)first * a.H + h;
    const size_t step = (size_t)a.H * a.ws_pitch;
    const float4 s0 = __ldcg(st), s1 = __ldcg(st + 1);
    float s[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
    constexpr int AHEAD = 4;
    for (int c = 0; c < chunks; c += AHEAD) {
        float4 m[AHEAD][2];
        float f[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c + j >= chunks) break;
            f[j] = __ldcg(total + (size_t)(c + j) * a.H);
            m[j][0] = __ldcg(reinterpret_cast<const float4*>(w + (size_t)(c + j) * step));
            m[j][1] = __ldcg(reinterpret_cast<const float4*>(w + (size_t)(c + j) * step) + 1);
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c + j >= chunks) break;
            uint4 hi, lo;
            split_pair(s[0], s[1], hi.x, lo.x);
            split_pair(s[2], s[3], hi.y, lo.y);
            split_pair(s[4], s[5], hi.z, lo.z);
            split_pair(s[6], s[7], hi.w, lo.w);
            reinterpret_cast<uint4*>(w + (size_t)(c + j) * step)[0] = hi;
            reinterpret_cast<uint4*>(w + (size_t)(c + j) * step)[1] = lo;
            const float mv[8] = {m[j][0].x, m[j][0].y, m[j][0].z, m[j][0].w, m[j][1].x, m[j][1].y, m[j][1].z, m[j][1].w};
#pragma unroll
            for (int i = 0; i < 8; ++i) s[i] = fmaf(f[j], s[i], mv[i]);
        }
    }
    st[0] = make_float4(s[0], s[1], s[2], s[3]);
    st[1] = make_float4(s[4], s[5], s[6], s[7]);
}

// grid (chunks, H / heads, value slabs). A warp owns 16 tokens of the chunk.
__global__ void __launch_bounds__(SC_THREADS) ssm_chunk_outputs_kernel(SsmChunkArgs a) {
    extern __shared__ __align__(128) unsigned char smem_raw[];
    const int NP = (a.N + 15) / 16 * 16, pitch = NP + 8, h0 = blockIdx.y * a.heads, v0 = blockIdx.z * SC_VALUES, group = h0 / a.per_group;
    bf16* cs = reinterpret_cast<bf16*>(smem_raw);        // [64][pitch]
    bf16* ss = cs + CHUNK_TOKENS * pitch;                // the state: [NP][SC_S_PITCH], hi and lo of eight columns in turn; at first B [64][pitch]
    bf16* xs = ss + (size_t)max(NP * SC_S_PITCH, CHUNK_TOKENS * pitch);          // [2][64][SC_X_PITCH]
    __shared__ Decays dec[SC_MAX_HEADS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mat = lane >> 3, r = lane & 7, g = lane >> 2, t = lane & 3;
    int t0 = 0, count = 0;
    pdl_enter();
    if (!chunk_of(a.cu_seqlens, a.B, blockIdx.x, t0, count)) return;
    auto fetch_x = [&](int i) { stage_rows(a, xs + (i & 1) * CHUNK_TOKENS * SC_X_PITCH, SC_X_PITCH, a.x_off + (h0 + i) * a.V + v0, SC_VALUES, a.V - v0, t0, count); };
    auto fetch_state = [&](int i) {
        const unsigned char* src = reinterpret_cast<const unsigned char*>(a.ws + ((size_t)blockIdx.x * a.H + h0 + i) * a.ws_pitch + v0);
        constexpr int PER = 2 * SC_VALUES / 8;           // 16-byte pieces of a row
        for (int e = threadIdx.x; e < NP * PER; e += SC_THREADS) {
            const int n = e / PER, c = e % PER;
            bf16* to = ss + n * SC_S_PITCH + c * 8;
            if (n < a.N && v0 + (c >> 1) * 8 < a.V) cp_async16(smem_u32(to), src + (size_t)n * a.V * 4 + c * 16);
            else *reinterpret_cast<uint4*>(to) = make_uint4(0u, 0u, 0u, 0u);
        }
    };
    stage_rows(a, cs, pitch, a.c_off + group * a.N, NP, a.N, t0, count);
    stage_rows(a, ss, pitch, a.b_off + group * a.N, NP, a.N, t0, count);
    cp_async_commit();
    load_decays(a, dec, h0, t0, count);
    cp_async_wait<0>();
    __syncthreads();
    // C B^T of the warp's 16 tokens with the chunk's 64, shared by the block's heads.
    float gm[8][4];
#pragma unroll
    for (int c = 0; c < 8; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) gm[c][e] = 0.f;
    const bf16* c_row = cs + (warp * 16 + (mat & 1) * 8 + r) * pitch + (mat >> 1) * 8;
    for (int ks = 0; ks < NP / 16; ++ks) {
        unsigned af[4];
        ldmatrix_x4(af, smem_u32(c_row + ks * 16));
#pragma unroll
        for (int np = 0; np < 4; ++np) {
            if (np > warp) break;                        // later tokens than the warp's own
            unsigned kb[4];
            ldmatrix_x4(kb, smem_u32(ss + (np * 16 + (mat >> 1) * 8 + r) * pitch + ks * 16 + (mat & 1) * 8));
            mma16816(gm[2 * np], af, kb[0], kb[1]);
            mma16816(gm[2 * np + 1], af, kb[2], kb[3]);
        }
    }
    __syncthreads();                                     // B is done with: the states take its place
    fetch_state(0);
    fetch_x(0);
    cp_async_commit();
    const int ta = warp * 16 + g, tb = ta + 8;
    for (int i = 0; i < a.heads; ++i) {
        const Decays& d = dec[i];
        cp_async_wait<0>();
        __syncthreads();
        float acc[8][4];
#pragma unroll
        for (int c = 0; c < 8; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[c][e] = 0.f;
        for (int ks = 0; ks < NP / 16; ++ks) {
            unsigned af[4];
            ldmatrix_x4(af, smem_u32(c_row + ks * 16));
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                unsigned vb[4];
                ldmatrix_x4_trans(vb, smem_u32(ss + (ks * 16 + (mat & 1) * 8 + r) * SC_S_PITCH + (2 * c + (mat >> 1)) * 8));
                mma16816(acc[c], af, vb[0], vb[1]);
                mma16816(acc[c], af, vb[2], vb[3]);
            }
        }
        const float pa = exp2f(d.hi[ta] + d.lo[ta]), pb = exp2f(d.hi[tb] + d.lo[tb]);
#pragma unroll
        for (int c = 0; c < 8; ++c) { acc[c][0] *= pa; acc[c][1] *= pa; acc[c][2] *= pb; acc[c][3] *= pb; }
        __syncthreads();                                 // the state is done with
        if (i + 1 < a.heads) {
            fetch_state(i + 1);
            fetch_x(i + 1);
            cp_async_commit();
        }
        const bf16* x = xs + (i & 1) * CHUNK_TOKENS * SC_X_PITCH;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk > warp) break;
            float p[2][4];
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int s = kk * 16 + q * 8 + 2 * t + (e & 1), tok = e < 2 ? ta : tb;
                    p[q][e] = s <= tok ? gm[2 * kk + q][e] * (d.dt[s] * decay_between(d, tok, s)) : 0.f;
                }
            unsigned ph[4], pl[4];
            split_pair(p[0][0], p[0][1], ph[0], pl[0]);
            split_pair(p[0][2], p[0][3], ph[1], pl[1]);
            split_pair(p[1][0], p[1][1], ph[2], pl[2]);
            split_pair(p[1][2], p[1][3], ph[3], pl[3]);
#pragma unroll
            for (int c = 0; c < 8; c += 2) {
                unsigned vb[4];
                ldmatrix_x4_trans(vb, smem_u32(x + (kk * 16 + (mat & 1) * 8 + r) * SC_X_PITCH + (c + (mat >> 1)) * 8));
                mma16816(acc[c], ph, vb[0], vb[1]);
                mma16816(acc[c], pl, vb[0], vb[1]);
                mma16816(acc[c + 1], ph, vb[2], vb[3]);
                mma16816(acc[c + 1], pl, vb[2], vb[3]);
            }
        }
        const float dh = a.skip[h0 + i];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int tok = half ? tb : ta;
            if (tok >= count) continue;
            float* out = a.y + (size_t)(t0 + tok) * a.H * a.V + (size_t)(h0 + i) * a.V + v0;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                if (v0 + c * 8 >= a.V) continue;
                const unsigned xv = *reinterpret_cast<const unsigned*>(x + tok * SC_X_PITCH + c * 8 + 2 * t);
                *reinterpret_cast<float2*>(out + c * 8 + 2 * t) = make_float2(fmaf(dh, __uint_as_float(xv << 16), acc[c][2 * half]),
                                                                              fmaf(dh, __uint_as_float(xv & 0xffff0000u), acc[c][2 * half + 1]));
            }
        }
    }
}

extern "C" int ti_memory_chunk_pitch(int D, int V);

// bfloat16 rows of state sizes up to 256 and value sizes in steps of 8; arguments as ti_ssm_chunks. Returns 2 for sizes outside that (the
// caller then takes ti_ssm_chunks).
extern "C" int ti_ssm_chunks_tc(float* o, const void* rows, long long ld, int x_off, int b_off, int c_off, float* state, long long state_stride,
                                const float* coef, const float* skip, float* ws, float* total, int chunks, const int* cu_seqlens, const int* seq_slots,
                                int B, int H, int groups, int N, int V, cudaStream_t stream) {
    if (B == 0 || chunks == 0) return 0;
    TI_REQUIRE(H > 0 && groups > 0 && H % groups == 0 && N > 0 && V > 0 && H <= 65535 && B <= 65535, "ssm_chunks_tc: %d heads in %d groups, %d x %d", H, groups, N, V);
    if (N % 8 != 0 || N > 256 || V % 8 != 0 || ld % 8 != 0 || x_off % 8 != 0 || b_off % 8 != 0 || c_off % 8 != 0 || state_stride % 4 != 0 || !aligned16(rows) ||
        !aligned16(state) || !aligned16(ws) || !aligned16(o)) {
        ti_fail("ssm_chunks_tc takes state sizes up to 256 and value sizes in steps of 8; got %d x %d", N, V);
        return 2;
    }
    const int per_group = H / groups, v_slabs = (V + SC_VALUES - 1) / SC_VALUES, n_slabs = (N + SC_ROWS - 1) / SC_ROWS;
    int heads = SC_MAX_HEADS;                            // as many heads a block as still fill the device
    while (heads > 1 && (per_group % heads != 0 || (long long)chunks * (H / heads) * v_slabs < 2LL * ti_sm_count())) heads >>= 1;
    const SsmChunkArgs a = {(const bf16*)rows, ld, x_off, b_off, c_off, coef, skip, cu_seqlens, B, H, per_group, heads, N, V, ws, ti_memory_chunk_pitch(N, V), total, o};
    const int NP = (N + 15) / 16 * 16, top = NP < SC_ROWS ? NP : SC_ROWS;
    const size_t smem_s = (size_t)CHUNK_TOKENS * (top + 8 + 2 * SC_X_PITCH) * sizeof(bf16);
    const size_t s_elems = (size_t)NP * SC_S_PITCH > (size_t)CHUNK_TOKENS * (NP + 8) ? (size_t)NP * SC_S_PITCH : (size_t)CHUNK_TOKENS * (NP + 8);
    const size_t smem_o = ((size_t)CHUNK_TOKENS * (NP + 8) + s_elems + 2 * CHUNK_TOKENS * SC_X_PITCH) * sizeof(bf16);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(ssm_chunk_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(ssm_chunk_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
        if (e != cudaSuccess) return ti_fail("ssm_chunks_tc: %s", cudaGetErrorString(e));
        configured = true;
    }
    ti_launch(ssm_chunk_states_kernel, dim3(chunks, H / heads, n_slabs * v_slabs), dim3(SC_THREADS), smem_s, stream, a);
    if (int rc = ti_check_launch("ssm_chunk_states")) return rc;
    ti_launch(ssm_chunk_scan_kernel, dim3((N * V / 8 + 127) / 128, H, B), dim3(128), 0, stream, a, state, state_stride, seq_slots);
    if (int rc = ti_check_launch("ssm_chunk_scan")) return rc;
    ti_launch(ssm_chunk_outputs_kernel, dim3(chunks, H / heads, v_slabs), dim3(SC_THREADS), smem_o, stream, a);
    return ti_check_launch("ssm_chunk_outputs");
}
