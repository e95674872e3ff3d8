// A 32-bit residual stream whose sublayers are added through a learned gate, normed in groups, with a short causal convolution over
// time ahead of a mixer.
//
//   gated_add_norm32   x += mult * (d + bias) * sigmoid(g + gbias);  h = T(G(x) * w), G: the row in `groups` equal parts, each divided by
//                      its own sqrt(mean(part^2) + eps) (`offset`: times 1 + w);  for one-token steps also hc = T(h + conv(h)) from and to the sequences' history
//   pair_add_norm32    the same for two sublayers side by side, each normed over the row first:
//                      x += mult * (sa A / rms(A) * wa + sb B / rms(B) * wb);  h = T(x / rms(x) * w)
//   conv_rows          hc = T(h + conv(h)), conv(h)_t = sum_j c[j] * h_(t - taps + 1 + j) per channel, over a step's rows (rows before the
//                      step from the history; its update is history_update, a launch of its own, since these blocks read it)
//
// d (the sublayer's output): rows [n, size] of T, 32-bit partial sums [s, n, size], or rows still apart: row t is
// sum_j scores[t, j] * d[index[t, j]] (the units a token went through). g: rows or partial sums. Everything between the loads and the
// one rounding on store is 32-bit; conv reads h as it was rounded, so that a row from the history equals a row of the step.
#include "common.cuh"

#define CONV_MAX_TAPS 64

struct BranchRows {                     // one of: rows, partials, rows with an index
    const void* rows;
    const float* partials;
    int n_partials;
    long long stride;
    const int* index;
    const float* scores;
    int per_row;
    const void* bias;
};
struct ConvStep {                       // conv [taps][size] of T (null: none); hist [slots][taps - 1][size] float, hist_stride floats a slot
    const void* conv;
    int taps;
    float* hist;
    long long hist_stride;
    const int* seq_slots;
    void* out;
};

template <typename T, int VEC> struct Piece {           // VEC neighbouring elements of a row of T or of float
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

template <typename T, int VEC>
__device__ __forceinline__ void branch_piece(const BranchRows& b, int row, int size, int i, float (&v)[VEC]) {
    if (b.partials != nullptr) {
        const float* p = b.partials + (size_t)row * size + i;
        Piece<float, VEC>::load(p, v);
        for (int s = 1; s < b.n_partials; ++s) {
            float u[VEC];
            Piece<float, VEC>::load(p + (size_t)s * b.stride, u);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] += u[e];
        }
    } else if (b.index != nullptr) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = 0.f;
        for (int j = 0; j < b.per_row; ++j) {
            const int r = __ldcg(b.index + (size_t)row * b.per_row + j);
            const float s = __ldcg(b.scores + (size_t)row * b.per_row + j);
            float u[VEC];
            Piece<T, VEC>::load((const T*)b.rows + (size_t)r * size + i, u);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = fmaf(s, u[e], v[e]);
        }
    } else {
        Piece<T, VEC>::load((const T*)b.rows + (size_t)row * b.stride + i, v);
    }
    if (b.bias != nullptr) {
        float u[VEC];
        Piece<T, VEC>::load((const T*)b.bias + i, u);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] += u[e];
    }
}

template <typename T, int VEC>
__global__ void gated_add_norm32_kernel(float* x, BranchRows d, BranchRows g, T* h, const T* __restrict__ w, float eps, int groups, ConvStep cs,
                                        int size, int has_branch, int has_gate, float mult, int offset) {
    extern __shared__ __align__(16) float row_d[];       // [size] the stream's new row, then [groups] sums' reciprocals, then partial sums
    const int row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    float* xr = x + (size_t)row * size;
    float* inv = row_d + (size + 3) / 4 * 4;
    float* sums = inv + groups;
    pdl_enter();
    for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
        float v[VEC];
        Piece<float, VEC>::load(xr + i, v);
        if (has_branch) {
            float dv[VEC];
            branch_piece<T, VEC>(d, row, size, i, dv);
            if (has_gate) {
                float gv[VEC];
                branch_piece<T, VEC>(g, row, size, i, gv);
#pragma unroll
                for (int e = 0; e < VEC; ++e) dv[e] = dv[e] / (1.0f + expf(-gv[e]));
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = fmaf(mult, dv[e], v[e]);
            Piece<float, VEC>::store(xr + i, v);
        }
        Piece<float, VEC>::store(row_d + i, v);
    }
    if (h == nullptr) return;
    __syncthreads();
    // The groups' sums of squares: `team` warps share a group where there are fewer groups than warps; the order of a group's sum
    // depends on the row's size and the number of groups alone.
    const int per = size / groups, team = warps > groups ? warps / groups : 1, teams = warps / team;
    if (warp < teams * team)
        for (int q = warp / team; q < groups; q += teams) {
            float ss = 0.f;
            for (int i = (warp % team) * 32 + lane; i < per; i += team * 32) {
                const float v = row_d[q * per + i];
                ss = fmaf(v, v, ss);
            }
            ss = warp_sum(ss);
            if (lane == 0) sums[q * team + warp % team] = ss;
        }
    __syncthreads();
    for (int q = threadIdx.x; q < groups; q += blockDim.x) {
        float ss = 0.f;
        for (int p = 0; p < team; ++p) ss += sums[q * team + p];
        inv[q] = 1.0f / sqrtf(ss / (float)per + eps);
    }
    __syncthreads();
    float* hist = cs.conv != nullptr && cs.taps > 1 ? cs.hist + (size_t)__ldcg(cs.seq_slots + row) * cs.hist_stride : nullptr;
    for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
        float v[VEC], wv[VEC];
        Piece<T, VEC>::load(w + i, wv);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = rnd<T>(row_d[i + e] * inv[(i + e) / per] * (offset ? 1.0f + wv[e] : wv[e]));
        Piece<T, VEC>::store(h + (size_t)row * size + i, v);
        if (cs.conv == nullptr) continue;
        // One token per sequence: row r is sequence r's token. A thread owns its channels' history: it reads and moves it on.
        float acc[VEC], c[VEC], u[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
        for (int j = 0; j < cs.taps - 1; ++j) {
            Piece<float, VEC>::load(hist + (size_t)j * size + i, u);
            Piece<T, VEC>::load((const T*)cs.conv + (size_t)j * size + i, c);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] = fmaf(c[e], u[e], acc[e]);
            if (j > 0) Piece<float, VEC>::store(hist + (size_t)(j - 1) * size + i, u);
        }
        Piece<T, VEC>::load((const T*)cs.conv + (size_t)(cs.taps - 1) * size + i, c);
        if (hist != nullptr) Piece<float, VEC>::store(hist + (size_t)(cs.taps - 2) * size + i, v);
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = v[e] + fmaf(c[e], v[e], acc[e]);
        Piece<T, VEC>::store((T*)cs.out + (size_t)row * size + i, acc);
    }
}

static int row_vec_ok(const BranchRows& b, int elem) {
    const uintptr_t mask = elem == 2 ? 7 : 15;
    return (((uintptr_t)b.rows | (uintptr_t)b.bias) & mask) == 0 && aligned16(b.partials) && b.stride % 4 == 0;
}

// The branch d (rows with a stride of d_stride elements between rows, or `d_partials` with d_stride floats between parts, or rows with
// index and scores [n, per_row]) and its bias [size] may be absent (then x is only normed), and so may the gate. h null: the stream's
// update alone. conv null: no convolution.
extern "C" int ti_gated_add_norm32(float* x, const void* d, const float* d_partials, int d_n, long long d_stride, const int* index, const float* scores,
                                   int per_row, const void* d_bias, const void* g, const float* g_partials, int g_n, long long g_stride,
                                   const void* g_bias, float mult, void* h, const void* w, int offset, float eps, int groups, const void* conv, int taps, float* hist,
                                   long long hist_stride, const int* seq_slots, void* conv_out, int n_rows, int size, int dtype, cudaStream_t stream) {
    if (n_rows == 0) return 0;
    TI_REQUIRE(size > 0 && size <= 40000 && groups >= 1 && groups <= 4096 && size % groups == 0, "gated_add_norm32: rows of %d in %d groups", size, groups);
    TI_REQUIRE(d == nullptr || d_partials == nullptr, "gated_add_norm32: the branch is rows or partial sums");
    TI_REQUIRE(index == nullptr || (d != nullptr && scores != nullptr && per_row >= 1), "gated_add_norm32: gathered rows need their rows, scores and a count");
    TI_REQUIRE(g == nullptr || g_partials == nullptr, "gated_add_norm32: the gate is rows or partial sums");
    TI_REQUIRE(conv == nullptr || (h != nullptr && conv_out != nullptr && taps >= 1 && taps <= CONV_MAX_TAPS && (taps == 1 || (hist != nullptr && seq_slots != nullptr))),
               "gated_add_norm32: a convolution of %d taps", taps);
    TI_REQUIRE(h == nullptr || w != nullptr, "gated_add_norm32: the norm needs its weight");
    const BranchRows db = {d, d_partials, d_n, d_stride, index, scores, per_row, d_bias}, gb = {g, g_partials, g_n, g_stride, nullptr, nullptr, 0, g_bias};
    const ConvStep cs = {conv, taps, hist, hist_stride, seq_slots, conv_out};
    const int has_branch = d != nullptr || d_partials != nullptr, has_gate = g != nullptr || g_partials != nullptr;
    const int threads = size >= 4096 ? 512 : size >= 1024 ? 256 : 128;
    const size_t smem = (size_t)((size + 3) / 4 * 4 + groups + (groups > threads / 32 ? groups : threads / 32)) * sizeof(float);
    TI_DISPATCH_DTYPE(dtype, {
        const uintptr_t mask = sizeof(T) == 2 ? 7 : 15;
        const bool vec = size % 4 == 0 && aligned16(x) && (((uintptr_t)h | (uintptr_t)w | (uintptr_t)conv | (uintptr_t)conv_out) & mask) == 0 &&
                         aligned16(hist) && hist_stride % 4 == 0 && row_vec_ok(db, sizeof(T)) && row_vec_ok(gb, sizeof(T));
        if (smem > 48 * 1024) {
            cudaFuncSetAttribute(gated_add_norm32_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            cudaFuncSetAttribute(gated_add_norm32_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        }
        if (vec) ti_launch(gated_add_norm32_kernel<T, 4>, dim3(n_rows), dim3(threads), smem, stream, x, db, gb, (T*)h, (const T*)w, eps, groups, cs, size, has_branch, has_gate, mult, offset);
        else ti_launch(gated_add_norm32_kernel<T, 1>, dim3(n_rows), dim3(threads), smem, stream, x, db, gb, (T*)h, (const T*)w, eps, groups, cs, size, has_branch, has_gate, mult, offset);
    });
    return ti_check_launch("gated_add_norm32");
}

// ------------------------------------------------------------------------------------------------ two sublayers at once
struct PairSum {
    BranchRows a, b;
    const void* wa;
    const void* wb;
    float sa, sb, eps;
};
template <typename T, int VEC>
__global__ void pair_add_norm32_kernel(float* x, PairSum p, T* __restrict__ h, const T* __restrict__ w, float eps, float mult, int offset, int size) {
    extern __shared__ __align__(16) float rows[];        // [2][size]: A and B, then the stream's new row
    __shared__ float scratch[33];
    const int row = blockIdx.x, padded = (size + 3) / 4 * 4;
    float* xr = x + (size_t)row * size;
    float ssa = 0.f, ssb = 0.f, ss = 0.f;
    pdl_enter();
    for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
        float va[VEC], vb[VEC];
        branch_piece<T, VEC>(p.a, row, size, i, va);
        branch_piece<T, VEC>(p.b, row, size, i, vb);
#pragma unroll
        for (int e = 0; e < VEC; ++e) { ssa = fmaf(va[e], va[e], ssa); ssb = fmaf(vb[e], vb[e], ssb); }
        Piece<float, VEC>::store(rows + i, va);
        Piece<float, VEC>::store(rows + padded + i, vb);
    }
    const float ia = p.sa / sqrtf(block_sum(ssa, scratch) / (float)size + p.eps), ib = p.sb / sqrtf(block_sum(ssb, scratch) / (float)size + p.eps);
    for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {       // (a thread reads back the elements it wrote)
        float v[VEC], wa[VEC], wb[VEC];
        Piece<float, VEC>::load(xr + i, v);
        Piece<T, VEC>::load((const T*)p.wa + i, wa);
        Piece<T, VEC>::load((const T*)p.wb + i, wb);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            v[e] = fmaf(mult, fmaf(rows[i + e] * ia, wa[e], rows[padded + i + e] * ib * wb[e]), v[e]);
            ss = fmaf(v[e], v[e], ss);
        }
        Piece<float, VEC>::store(xr + i, v);
        Piece<float, VEC>::store(rows + i, v);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)size + eps);
    for (int i = threadIdx.x * VEC; i < size; i += blockDim.x * VEC) {
        float v[VEC], wv[VEC];
        Piece<T, VEC>::load(w + i, wv);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = rows[i + e] * inv * (offset ? 1.0f + wv[e] : wv[e]);
        Piece<T, VEC>::store(h + (size_t)row * size + i, v);
    }
}

// a, b: rows [n, size] with a stride, or partial sums with floats between parts, as ti_gated_add_norm32 takes them; wa, wb, w [size] of T.
extern "C" int ti_pair_add_norm32(float* x, const void* a, const float* a_partials, int a_n, long long a_stride, const void* b, const float* b_partials, int b_n,
                                  long long b_stride, const void* wa, const void* wb, float sa, float sb, float pair_eps, float mult, void* h, const void* w,
                                  int offset, float eps, int n_rows, int size, int dtype, cudaStream_t stream) {
    if (n_rows == 0) return 0;
    TI_REQUIRE(size > 0 && size <= 20000, "pair_add_norm32: rows of %d", size);
    TI_REQUIRE((a != nullptr) != (a_partials != nullptr) && (b != nullptr) != (b_partials != nullptr), "pair_add_norm32: each side is rows or partial sums");
    TI_REQUIRE(wa != nullptr && wb != nullptr && w != nullptr && h != nullptr, "pair_add_norm32: the norms need their weights");
    const PairSum p = {{a, a_partials, a_n, a_stride, nullptr, nullptr, 0, nullptr}, {b, b_partials, b_n, b_stride, nullptr, nullptr, 0, nullptr}, wa, wb, sa, sb, pair_eps};
    const int threads = size >= 4096 ? 512 : size >= 1024 ? 256 : 128;
    const size_t smem = (size_t)2 * ((size + 3) / 4 * 4) * sizeof(float);
    TI_DISPATCH_DTYPE(dtype, {
        const uintptr_t mask = sizeof(T) == 2 ? 7 : 15;
        const bool vec = size % 4 == 0 && aligned16(x) && (((uintptr_t)h | (uintptr_t)w | (uintptr_t)wa | (uintptr_t)wb) & mask) == 0 && row_vec_ok(p.a, sizeof(T)) &&
                         row_vec_ok(p.b, sizeof(T));
        if (smem > 48 * 1024) {
            cudaFuncSetAttribute(pair_add_norm32_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            cudaFuncSetAttribute(pair_add_norm32_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        }
        if (vec) ti_launch(pair_add_norm32_kernel<T, 4>, dim3(n_rows), dim3(threads), smem, stream, x, p, (T*)h, (const T*)w, eps, mult, offset, size);
        else ti_launch(pair_add_norm32_kernel<T, 1>, dim3(n_rows), dim3(threads), smem, stream, x, p, (T*)h, (const T*)w, eps, mult, offset, size);
    });
    return ti_check_launch("pair_add_norm32");
}

// ------------------------------------------------------------------------------------------------ the convolution over a step's rows
#define CR_TOKENS 16
// A thread owns VEC channels and walks a few rows; with the number of taps known at compile time (TAPS > 0) the rows before the current
// one stay in registers. A row's sum is taken in the order of the taps either way.
template <typename T, int VEC, int TAPS>
__global__ void conv_rows_kernel(T* __restrict__ out, const T* h, const T* __restrict__ conv, int taps, const float* hist, long long hist_stride,
                                 const int* cu_seqlens, const int* seq_slots, int B, int n, int size) {
    const int i = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    const int first = blockIdx.y * CR_TOKENS, last = min(n, first + CR_TOKENS);
    constexpr int BACK = TAPS > 0 ? TAPS - 1 : 0;
    float c[TAPS > 0 ? TAPS : 1][VEC], w[BACK > 0 ? BACK : 1][VEC];          // weights; the rows before the current one, oldest first
    if (TAPS > 0 && i < size)
#pragma unroll
        for (int j = 0; j < TAPS; ++j) Piece<T, VEC>::load(conv + (size_t)j * size + i, c[j]);
    pdl_enter();
    if (i >= size) return;
    int lo = 0, hi = B - 1;                              // the sequence of the first row: the last b with cu[b] <= first
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (__ldcg(cu_seqlens + mid) <= first) lo = mid; else hi = mid - 1;
    }
    int b = lo, begin = __ldcg(cu_seqlens + b), end = __ldcg(cu_seqlens + b + 1);
    auto earlier = [&](int r, float (&u)[VEC]) {         // row r of the step, or, ahead of the sequence's first, a row of its history
        if (r >= begin) Piece<T, VEC>::load(h + (size_t)r * size + i, u);
        else Piece<float, VEC>::load(hist + (size_t)__ldcg(seq_slots + b) * hist_stride + (size_t)(taps - 1 + r - begin) * size + i, u);
    };
    bool fresh = true;
    for (int t = first; t < last; ++t) {
        while (t >= end) { ++b; begin = end; end = __ldcg(cu_seqlens + b + 1); fresh = true; }
        float acc[VEC], v[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
        Piece<T, VEC>::load(h + (size_t)t * size + i, v);
        if constexpr (TAPS > 0) {
            if (fresh) {
#pragma unroll
                for (int j = 0; j < BACK; ++j) earlier(t - BACK + j, w[j]);
                fresh = false;
            }
#pragma unroll
            for (int j = 0; j < BACK; ++j)
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[e] = fmaf(c[j][e], w[j][e], acc[e]);
#pragma unroll
            for (int j = 0; j + 1 < BACK; ++j)
#pragma unroll
                for (int e = 0; e < VEC; ++e) w[j][e] = w[j + 1][e];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                if (BACK > 0) w[BACK > 0 ? BACK - 1 : 0][e] = v[e];
                acc[e] = v[e] + fmaf(c[BACK][e], v[e], acc[e]);
            }
        } else {
            float u[VEC], k[VEC];
            for (int j = 0; j < taps - 1; ++j) {
                earlier(t - (taps - 1) + j, u);
                Piece<T, VEC>::load(conv + (size_t)j * size + i, k);
#pragma unroll
                for (int e = 0; e < VEC; ++e) acc[e] = fmaf(k[e], u[e], acc[e]);
            }
            Piece<T, VEC>::load(conv + (size_t)(taps - 1) * size + i, k);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] = v[e] + fmaf(k[e], v[e], acc[e]);
        }
        Piece<T, VEC>::store(out + (size_t)t * size + i, acc);
    }
}

// out, h [n, size] of T; conv [taps, size]; hist [slots][taps - 1][size] float (hist_stride floats a slot; null with one tap).
extern "C" int ti_conv_rows(void* out, const void* h, const void* conv, int taps, const float* hist, long long hist_stride, const int* cu_seqlens,
                            const int* seq_slots, int n, int B, int size, int dtype, cudaStream_t stream) {
    if (n == 0) return 0;
    TI_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS && (taps == 1 || hist != nullptr) && B >= 1, "conv_rows: %d taps", taps);
#define CR_LAUNCH(TAPS)                                                                                                                                     \
    do {                                                                                                                                                    \
        if (vec) ti_launch(conv_rows_kernel<T, 4, TAPS>, grid, dim3(threads), 0, stream, (T*)out, (const T*)h, (const T*)conv, taps, hist, hist_stride, cu_seqlens, seq_slots, B, n, size); \
        else ti_launch(conv_rows_kernel<T, 1, TAPS>, grid, dim3(threads), 0, stream, (T*)out, (const T*)h, (const T*)conv, taps, hist, hist_stride, cu_seqlens, seq_slots, B, n, size); \
    } while (0)
    TI_DISPATCH_DTYPE(dtype, {
        const uintptr_t mask = sizeof(T) == 2 ? 7 : 15;
        const bool vec = size % 4 == 0 && (((uintptr_t)out | (uintptr_t)h | (uintptr_t)conv) & mask) == 0 && aligned16(hist) && hist_stride % 4 == 0;
        const int per = vec ? 4 : 1, threads = 128;
        const dim3 grid((size / per + threads - 1) / threads, (n + CR_TOKENS - 1) / CR_TOKENS);
        switch (taps) {
            case 1: CR_LAUNCH(1); break;
            case 2: CR_LAUNCH(2); break;
            case 3: CR_LAUNCH(3); break;
            case 4: CR_LAUNCH(4); break;
            default: CR_LAUNCH(0); break;
        }
    });
#undef CR_LAUNCH
    return ti_check_launch("conv_rows");
}
