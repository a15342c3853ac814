// Gated linear attention: the scan's instances (channel_memory.cuh).  Its records come from low_rank.cu.
#include "channel_memory.cuh"

extern "C" {

// rec [H, T, 3 Kp]; y [T, H V] receives S^T q times q_scale; S [H, V, K] at s_off of the requests' state moves on.
int infero_decayed_scan(const float* rec, int n_tokens, const float* v, long long v_stride, float q_scale, float* state,
                        long long state_stride, long long s_off, const int* entry_q_start, const int* entry_q_len, const int* entry_slot,
                        float* y, int n_entries, int single, int H, int K, int V, int sm_count, cudaStream_t stream) {
    return memory::channel_scan<false>(rec, n_tokens, v, v_stride, state, state_stride, s_off, entry_q_start, entry_q_len, entry_slot, y,
                                       q_scale, n_entries, single, H, K, V, sm_count, stream);
}

}  // extern "C"
