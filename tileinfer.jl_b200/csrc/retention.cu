// Retention: linear attention with a fixed decay per head whose q and k are rotated by the token's position,
//
//   S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   q, k <- rotation(q), rotation(k) times q_scale, k_scale
//
// over the tokens a step brings, from and to a 32-bit state per (sequence, head). The scan itself is lightning_scan.cuh's; rotation and
// scales are 32-bit and are not rounded before the recurrence. One-token steps run in matrix_memory.cu's memory_token.
#include "lightning_scan.cuh"

// qkv [n, ld] of T with the heads' queries from column q_off on (H * D of them), keys from k_off, values from v_off (H * V); a
// sequence's state [H, D, V] float at slot * state_stride; cos_sin [positions, rotary / 2, 2] float or null; positions [n].
extern "C" int ti_retention_scan(float* o, const void* qkv, long long ld, int q_off, int k_off, int v_off, float* state, long long state_stride,
                                 const float* decay, const float* cos_sin, int rotary, const int* positions, float q_scale, float k_scale,
                                 const int* cu_seqlens, const int* seq_slots, int n_tokens, int B, int H, int D, int V, int dtype,
                                 cudaStream_t stream) {
    if (B == 0) return 0;
    TI_REQUIRE(cos_sin == nullptr || (positions != nullptr && rotary >= 2 && rotary % 2 == 0 && rotary <= D), "retention_scan: rotation over %d of %d", rotary, D);
    ScanExtras ex = {};
    ex.state_stride = state_stride;
    ex.cos_sin = cos_sin; ex.rotary = rotary; ex.positions = positions;
    ex.q_scale = q_scale; ex.k_scale = k_scale;
    return launch_lightning_scan<1>("retention_scan", o, qkv, ld, q_off, k_off, v_off, state, decay, cu_seqlens, seq_slots, n_tokens, B, H, D, V, 0, ex,
                                    dtype, stream);
}
