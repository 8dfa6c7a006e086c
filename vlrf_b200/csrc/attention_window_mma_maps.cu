// The kernels of attention_window_mma.cuh for two maps a head (differential attention).
#include "common.cuh"
#include "attention_window_mma.cuh"

int attn_window_mma_two_maps(const void* q, int ldq, const void* Kc, const void* Vc, const int* block_table, int max_blocks, const int* seq_slot,
                             const int* seq_start, const int* seq_pos0, void* out, int ld_out, float* partials, int n_seqs, int max_new, int H,
                             int Hkv, int dk, int dv, float scale, int window, float out_scale, int n_split, float softcap, int keep_first,
                             const float* slopes, float map_factor, float head_eps, int* dev_err, cudaStream_t stream) {
    return window_mma_by_size<2>(q, ldq, Kc, Vc, block_table, max_blocks, seq_slot, seq_start, seq_pos0, out, ld_out, partials, n_seqs, max_new, H, Hkv,
                                 dk, dv, scale, window, out_scale, n_split, softcap, keep_first, nullptr, nullptr, 0, slopes, map_factor, head_eps,
                                 dev_err, stream);
}
