// Gated linear attention: the scan's instances.  See outer_memory.cu.
#include "outer_memory.cuh"

int memory::scan_decayed(const ScanArgs& a, int n_entries, bool single, int sm_count, cudaStream_t stream) {
    return launch_channel_scan<RULE_DECAYED>(a, n_entries, single, sm_count, stream);
}
