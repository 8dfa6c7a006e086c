// Attention with key and value sizes of their own on the tensor cores: the entry points, the kernels of one map a head, and
// the merges of a cut context's parts.  What is computed and how: attention_window_mma.cuh.
#include "common.cuh"
#include "attention_window_mma.cuh"

namespace {
// The parts of a decode step's contexts: out[row][h] = out_scale · Σ_p o_p 2^(m_p − M) / Σ_p l_p 2^(m_p − M), in the
// order of the parts.  A part that saw no key has l = 0.
__global__ void __launch_bounds__(128)
attn_window_merge_kernel(const float* __restrict__ partials, const int* __restrict__ seq_slot, __nv_bfloat16* __restrict__ out,
                         int ld_out, int H, int dv, int n_split, float out_scale, const float* __restrict__ sink,
                         const float* __restrict__ gate, int ld_gate) {
    pdl_wait();
    pdl_launch_dependents();
    const int row = blockIdx.x, h = blockIdx.y;
    if (seq_slot[row] < 0) return;
    const float* p = partials + ((size_t)row * H + h) * n_split * (dv + 2);
    float M = -INFINITY;
    for (int s = 0; s < n_split; ++s)
        if (p[s * (dv + 2) + dv + 1] > 0.f) M = fmaxf(M, p[s * (dv + 2) + dv]);
    const float sk = sink != nullptr ? sink[h] * 1.4426950408889634f : -INFINITY;
    M = fmaxf(M, sk);
    float L = sink != nullptr ? exp2f(sk - M) : 0.f;
    for (int s = 0; s < n_split; ++s) {
        const float l = p[s * (dv + 2) + dv + 1];
        if (l > 0.f) L += l * exp2f(p[s * (dv + 2) + dv] - M);
    }
    const float inv = (L > 0.f ? out_scale / L : 0.f) * (gate != nullptr ? sigmoid_f(gate[(size_t)row * ld_gate + h]) : 1.f);
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        float acc = 0.f;
        for (int s = 0; s < n_split; ++s)
            if (p[s * (dv + 2) + dv + 1] > 0.f) acc += p[s * (dv + 2) + c] * exp2f(p[s * (dv + 2) + dv] - M);
        out[(size_t)row * ld_out + (size_t)h * dv + c] = __float2bfloat16_rn(acc * inv);
    }
}

// The same for two maps: the second map's result times map_factor off the first's, then the head's dv numbers over their root
// mean square.  dv ≤ 128: a thread per column.
__global__ void __launch_bounds__(128)
attn_window_merge_maps_kernel(const float* __restrict__ partials, const int* __restrict__ seq_slot, __nv_bfloat16* __restrict__ out,
                              int ld_out, int H, int dv, int n_split, float out_scale, float map_factor, float head_eps) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float red[4];
    const int row = blockIdx.x, h = blockIdx.y, c = threadIdx.x;
    if (seq_slot[row] < 0) return;
    float x = 0.f;
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
        const float* p = partials + (((size_t)row * H + h) * 2 + mp) * n_split * (dv + 2);
        float M = -INFINITY, L = 0.f, acc = 0.f;
        for (int s = 0; s < n_split; ++s)
            if (p[s * (dv + 2) + dv + 1] > 0.f) M = fmaxf(M, p[s * (dv + 2) + dv]);
        for (int s = 0; s < n_split; ++s) {
            const float l = p[s * (dv + 2) + dv + 1];
            if (l > 0.f) {
                const float f = exp2f(p[s * (dv + 2) + dv] - M);
                L = fmaf(l, f, L);
                if (c < dv) acc = fmaf(p[s * (dv + 2) + c], f, acc);
            }
        }
        const float r = L > 0.f ? acc / L : 0.f;
        x = mp == 0 ? r : x - map_factor * r;
    }
    const float part = warp_sum(x * x);
    if ((c & 31) == 0) red[c >> 5] = part;
    __syncthreads();
    const float f = out_scale / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)dv + head_eps);
    if (c < dv) out[(size_t)row * ld_out + (size_t)h * dv + c] = __float2bfloat16_rn(x * f);
}
}  // namespace

// attention_window_mma_maps.cu
int attn_window_mma_two_maps(const void* q, int ldq, const void* Kc, const void* Vc, const int* block_table, int max_blocks, const int* seq_slot,
                             const int* seq_start, const int* seq_pos0, void* out, int ld_out, float* partials, int n_seqs, int max_new, int H,
                             int Hkv, int dk, int dv, float scale, int window, float out_scale, int n_split, float softcap, int keep_first,
                             const float* slopes, float map_factor, float head_eps, int* dev_err, cudaStream_t stream);

// Whether the tensor-core kernel takes these sizes (bfloat16 only): head sizes multiples of 8 up to 128, at most 16
// query heads a key/value head, cache blocks of 64 tokens, rows on 16-byte boundaries.
extern "C" int vlrf_attn_window_mma_takes(int H, int Hkv, int dk, int dv, int BT, int ldq, int ld_out) {
    return (H > 0 && Hkv > 0 && H % Hkv == 0 && H / Hkv <= 16 && dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 128 &&
            dv <= 128 && BT == WM_BK && ldq % 8 == 0 && ld_out % 2 == 0) ? 1 : 0;
}

extern "C" int vlrf_attn_window_mma_ex(const void* q, int ldq, const void* Kc, const void* Vc, const int* block_table, int max_blocks,
                                       const int* seq_slot, const int* seq_start, const int* seq_pos0, void* out, int ld_out,
                                       float* partials, int n_seqs, int max_new, int H, int Hkv, int dk, int dv, int BT, float scale,
                                       int window, float out_scale, int n_split, float softcap, int keep_first, const float* sink,
                                       const float* gate, int ld_gate, const float* slopes, int maps, float map_factor, float head_eps, int* dev_err,
                                       cudaStream_t stream) {
    VLRF_REQUIRE(maps == 1 || (maps == 2 && sink == nullptr && gate == nullptr && head_eps > 0.f),
                 "attn_window_mma: one map, or two without sinks and gates and with a positive eps");
    VLRF_REQUIRE(vlrf_attn_window_mma_takes(H, Hkv, dk, dv, BT, ldq, ld_out), "attn_window_mma: heads %d/%d, sizes %d and %d, block %d are not taken",
                 H, Hkv, dk, dv, BT);
    VLRF_REQUIRE(n_seqs >= 0 && max_new >= 0 && max_blocks > 0 && window >= 0 && dev_err != nullptr, "attn_window_mma: bad arguments");
    VLRF_REQUIRE(keep_first >= 0 && softcap >= 0.f && (gate == nullptr || ld_gate >= H), "attn_window_mma: negative kept tokens or cap, or gate rows shorter than the heads");
    VLRF_REQUIRE(n_seqs <= 65535 && Hkv <= 65535, "attn_window_mma: too many sequences or heads for one launch");
    VLRF_REQUIRE(n_split >= 1 && (n_split == 1 || (max_new == 1 && partials != nullptr)),
                 "attn_window_mma: contexts are cut into parts in decode steps only, and the parts need scratch");
    VLRF_REQUIRE((reinterpret_cast<uintptr_t>(q) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 3) == 0, "attn_window_mma: misaligned rows");
    if (n_seqs == 0 || max_new == 0) return VLRF_OK;
    const int st = maps == 2
        ? attn_window_mma_two_maps(q, ldq, Kc, Vc, block_table, max_blocks, seq_slot, seq_start, seq_pos0, out, ld_out, partials, n_seqs, max_new, H,
                                   Hkv, dk, dv, scale, window, out_scale, n_split, softcap, keep_first, slopes, map_factor, head_eps, dev_err, stream)
        : window_mma_by_size<1>(q, ldq, Kc, Vc, block_table, max_blocks, seq_slot, seq_start, seq_pos0, out, ld_out, partials, n_seqs, max_new, H, Hkv,
                                dk, dv, scale, window, out_scale, n_split, softcap, keep_first, sink, gate, ld_gate, slopes, 0.f, 1.f, dev_err, stream);
    if (st != VLRF_OK) return st;
    if (n_split > 1 && maps == 2) {
        launch_chained(attn_window_merge_maps_kernel, dim3(n_seqs, H), dim3(128), (size_t)0, stream, (const float*)partials, seq_slot,
                       (__nv_bfloat16*)out, ld_out, H, dv, n_split, out_scale, map_factor, head_eps);
        return vlrf_check_launch("attn_window_merge");
    }
    if (n_split > 1) {
        launch_chained(attn_window_merge_kernel, dim3(n_seqs, H), dim3(128), (size_t)0, stream, (const float*)partials, seq_slot,
                       (__nv_bfloat16*)out, ld_out, H, dv, n_split, out_scale, sink, gate, ld_gate);
        return vlrf_check_launch("attn_window_merge");
    }
    return VLRF_OK;
}

extern "C" int vlrf_attn_window_mma(const void* q, int ldq, const void* Kc, const void* Vc, const int* block_table, int max_blocks,
                                    const int* seq_slot, const int* seq_start, const int* seq_pos0, void* out, int ld_out,
                                    float* partials, int n_seqs, int max_new, int H, int Hkv, int dk, int dv, int BT, float scale,
                                    int window, float out_scale, int n_split, int* dev_err, cudaStream_t stream) {
    return vlrf_attn_window_mma_ex(q, ldq, Kc, Vc, block_table, max_blocks, seq_slot, seq_start, seq_pos0, out, ld_out, partials,
                                   n_seqs, max_new, H, Hkv, dk, dv, BT, scale, window, out_scale, n_split, 0.f, 0, nullptr, nullptr, 0,
                                   nullptr, 1, 0.f, 0.f, dev_err, stream);
}
