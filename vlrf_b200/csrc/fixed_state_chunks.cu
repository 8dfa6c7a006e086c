// The recurrence with a fixed decay per head over prompts, chunk by chunk on the tensor cores (`mma.sync`, bfloat16 inputs).
//
// A head keeps a matrix S of K rows by V columns, S ← a S + k vᵀ, o = Sᵀ q (matrix_state.cu, kind 3, which takes every size and the
// 32-bit engine).  Cut a sequence's new tokens into chunks of 64; with S_c the state ahead of chunk c (L tokens, numbered from 0)
//
//     o_i     = a^(i+1) · S_cᵀ q_i + Σ_(j ≤ i) a^(i−j) (q_i · k_j) v_j
//     S_(c+1) = a^L · S_c + U_c,     U_c = Σ_j a^(L−1−j) k_j v_jᵀ
//
// so three kernels do it, each with every chunk at the same time but for the short sum in the middle:
//   chunk_writes   U_c of every chunk: tiles of 64 state rows by 64 columns, a product over the chunk's tokens
//   chunk_states   a thread per four numbers of a state walks its sequence's chunks: S_c takes U_c's place, the last one is kept
//   chunk_outputs  the two products of o, a CTA per chunk, head and up to 128 columns
//
// What is 32-bit: decays and their powers, the sums, S and U.  Where one of them is an operand of an MMA (S, a^n k, and the faded
// scores a^(i−j) q·k) it enters as the sum of two bfloat16 numbers (16 bits of it); q, k and v come as bfloat16.
//
// Layouts: q, k [T][H·K], v [T][H·V] bfloat16 (column ranges of wider rows); y float32 [T][H·V]; scratch [slot][H][V][K] float32, the
// slots of sequence s beginning at seq_start[s] / 64 + s (T / 64 + sequences in all); the sequences' states as in matrix_state.cu:
// [slots][2][state_row], head by head [V][K], read from the copy of the parity of the position at the step's start and written to
// that of its end.
#include "common.cuh"

namespace {
constexpr int FC = 64;                              // tokens of a chunk
constexpr int FC_MAX_K = 256;

__device__ __forceinline__ uint32_t fc_sm(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
// 16 bytes, or zeros where there is nothing
__device__ __forceinline__ void fc_cp16(void* dst, const void* src, bool there) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(fc_sm(dst)), "l"(src), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ void fc_ldsm(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void fc_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void fc_ldsm_t2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void fc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two numbers as the sum of two pairs of bfloat16
__device__ __forceinline__ void fc_split(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
// a^n by squaring, n ≥ 0
__device__ __forceinline__ float fc_power(float a, int n) {
    float r = 1.f;
    for (; n > 0; n >>= 1, a *= a)
        if (n & 1) r *= a;
    return r;
}

struct FixedChunks {
    const __nv_bfloat16 *q, *k, *v;
    int ldq, ldk, ldv;
    const float* decay;
    float q_scale;
    float *scratch, *state, *y;
    int state_row, ldy;
    const int *seq_slot, *seq_start, *seq_pos0;
    int H, K, V;
};

// grid (chunks of the longest run, H · tiles of the state, sequences)
__global__ void __launch_bounds__(128)
chunk_writes_kernel(const FixedChunks A, int k_tiles, int v_tiles) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int LD = 64 + 8;                      // (16 bytes of padding keep ldmatrix off bank conflicts)
    __shared__ __align__(16) __nv_bfloat16 ks[FC * LD], kl[FC * LD], vs[FC * LD];
    __shared__ float pw[FC];
    const int s = blockIdx.z, c0 = blockIdx.x * FC;
    const int start = A.seq_start[s], n = A.seq_start[s + 1] - start;
    if (c0 >= n || A.seq_slot[s] < 0) return;
    const int L = min(FC, n - c0);
    const int tile = blockIdx.y % (k_tiles * v_tiles), h = blockIdx.y / (k_tiles * v_tiles);
    const int k0 = (tile % k_tiles) * 64, v0 = (tile / k_tiles) * 64;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    for (int i = tid; i < FC * 8; i += 128) {
        const int r = i >> 3, ch = (i & 7) * 8;
        const size_t row = (size_t)(start + c0 + (r < L ? r : 0));
        fc_cp16(ks + r * LD + ch, A.k + row * A.ldk + (size_t)h * A.K + (k0 + ch < A.K ? k0 + ch : 0), r < L && k0 + ch < A.K);
        fc_cp16(vs + r * LD + ch, A.v + row * A.ldv + (size_t)h * A.V + (v0 + ch < A.V ? v0 + ch : 0), r < L && v0 + ch < A.V);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (tid < FC) pw[tid] = tid < L ? fc_power(A.decay[h], L - 1 - tid) : 0.f;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int i = tid; i < FC * 32; i += 128) {      // a^(L−1−j) k_j in two halves
        const int r = i >> 5, ch = (i & 31) * 2;
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(ks + r * LD + ch);
        uint32_t hi, lo;
        fc_split(__low2float(x) * pw[r], __high2float(x) * pw[r], hi, lo);
        *reinterpret_cast<uint32_t*>(ks + r * LD + ch) = hi;
        *reinterpret_cast<uint32_t*>(kl + r * LD + ch) = lo;
    }
    __syncthreads();
    // warp w: state columns (values) v0 + 16 w … + 15 as MMA rows, 64 state rows (key channels) as MMA columns
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < FC / 16; ++kk) {
        uint32_t a[4];                              // (tokens 0-7, values 0-7), (tokens 0-7, values 8-15), then tokens 8-15
        fc_ldsm_t(a, fc_sm(vs + (kk * 16 + (lane & 7) + 8 * (lane >> 4)) * LD + warp * 16 + 8 * ((lane >> 3) & 1)));
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
            uint32_t b[4];
            const int at = (kk * 16 + (lane & 15)) * LD + (j + (lane >> 4)) * 8;
            fc_ldsm_t(b, fc_sm(ks + at));
            fc_mma(acc[j], a, b[0], b[1]);
            fc_mma(acc[j + 1], a, b[2], b[3]);
            fc_ldsm_t(b, fc_sm(kl + at));
            fc_mma(acc[j], a, b[0], b[1]);
            fc_mma(acc[j + 1], a, b[2], b[3]);
        }
    }
    float* dst = A.scratch + ((size_t)(start / FC + s + blockIdx.x) * A.H + h) * A.V * A.K;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int v = v0 + warp * 16 + (lane >> 2) + 8 * r;
        if (v >= A.V) continue;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int k = k0 + j * 8 + 2 * (lane & 3);
            if (k < A.K) *reinterpret_cast<float2*>(dst + (size_t)v * A.K + k) = make_float2(acc[j][2 * r], acc[j][2 * r + 1]);
        }
    }
}

// grid (quads of a sequence's states / 128, sequences)
__global__ void __launch_bounds__(128)
chunk_states_kernel(const FixedChunks A) {
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.y, slot = A.seq_slot[s];
    if (slot < 0) return;
    const int start = A.seq_start[s], n = A.seq_start[s + 1] - start, pos0 = A.seq_pos0[s];
    const size_t per_head = (size_t)A.V * A.K, all = per_head * A.H;
    const size_t i = 4 * ((size_t)blockIdx.x * 128 + threadIdx.x);
    if (i >= all || n <= 0) return;
    const float a = A.decay[i / per_head];
    const float* from = A.state + ((size_t)slot * 2 + (pos0 & 1)) * A.state_row;
    float* to = A.state + ((size_t)slot * 2 + ((pos0 + n) & 1)) * A.state_row;
    const int chunks = (n + FC - 1) / FC;
    const float whole = fc_power(a, FC), last = fc_power(a, n - (chunks - 1) * FC);
    float4 S = *reinterpret_cast<const float4*>(from + i);
    float* u = A.scratch + (size_t)(start / FC + s) * all + i;
    constexpr int AHEAD = 8;                        // chunks asked for together
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float4 U[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) U[j] = c0 + j < chunks ? *reinterpret_cast<const float4*>(u + (size_t)(c0 + j) * all) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c0 + j < chunks) {
                *reinterpret_cast<float4*>(u + (size_t)(c0 + j) * all) = S;
                const float f = c0 + j == chunks - 1 ? last : whole;
                S.x = fmaf(f, S.x, U[j].x); S.y = fmaf(f, S.y, U[j].y); S.z = fmaf(f, S.z, U[j].z); S.w = fmaf(f, S.w, U[j].w);
            }
        }
    }
    *reinterpret_cast<float4*>(to + i) = S;
}

// NT: tiles of 8 columns a warp (a CTA takes 32·NT columns of V).  grid (chunks of the longest run, H · column tiles, sequences)
template <int NT>
__global__ void __launch_bounds__(128)
chunk_outputs_kernel(const FixedChunks A, int v_tiles) {
    pdl_wait();
    pdl_launch_dependents();
    constexpr int VT = 32 * NT, VS = VT + 8, PS = FC + 8;
    extern __shared__ __align__(16) unsigned char fc_raw[];
    const int K16 = (A.K + 15) & ~15, KS = K16 + 8;  // (columns behind K are zeros)
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(fc_raw);        // [64][KS]
    __nv_bfloat16* ks = qs + FC * KS;                                    // [64][KS]
    __nv_bfloat16* vs = ks + FC * KS;                                    // [64][VS]
    __nv_bfloat16* ph = vs + FC * VS;                                    // [64][PS]: the faded scores, high halves
    __nv_bfloat16* pl = ph + FC * PS;                                    // … low halves
    float* pw = reinterpret_cast<float*>(pl + FC * PS);                  // [65]: powers of the decay
    const int s = blockIdx.z, c0 = blockIdx.x * FC;
    const int start = A.seq_start[s], n = A.seq_start[s + 1] - start;
    if (c0 >= n || A.seq_slot[s] < 0) return;
    const int L = min(FC, n - c0);
    const int h = blockIdx.y / v_tiles, v0 = (blockIdx.y - h * v_tiles) * VT;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int kch = K16 / 8;
    for (int i = tid; i < FC * kch; i += 128) {
        const int r = i / kch, ch = (i - r * kch) * 8;
        const bool there = r < L && ch < A.K;
        const size_t row = (size_t)(start + c0 + (r < L ? r : 0)), col = (size_t)h * A.K + (ch < A.K ? ch : 0);
        fc_cp16(qs + r * KS + ch, A.q + row * A.ldq + col, there);
        fc_cp16(ks + r * KS + ch, A.k + row * A.ldk + col, there);
    }
    for (int i = tid; i < FC * (VT / 8); i += 128) {
        const int r = i / (VT / 8), ch = (i - r * (VT / 8)) * 8;
        fc_cp16(vs + r * VS + ch, A.v + (size_t)(start + c0 + (r < L ? r : 0)) * A.ldv + (size_t)h * A.V + (v0 + ch < A.V ? v0 + ch : 0), r < L && v0 + ch < A.V);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (tid <= FC) pw[tid] = fc_power(A.decay[h], tid);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    {   // the scores of rows 16 w … + 15 with the keys up to them, faded and split
        float sc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
        for (int kk = 0; kk < K16 / 16; ++kk) {
            uint32_t a[4];
            fc_ldsm(a, fc_sm(qs + (warp * 16 + (lane & 15)) * KS + kk * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                if (j <= 2 * warp + 1) {            // (keys 8j … 8j+15: (keys lo, k lo), (keys lo, k hi), (keys hi, k lo), (keys hi, k hi))
                    uint32_t b[4];
                    fc_ldsm(b, fc_sm(ks + (j * 8 + (lane & 7) + 8 * (lane >> 4)) * KS + kk * 16 + 8 * ((lane >> 3) & 1)));
                    fc_mma(sc[j], a, b[0], b[1]);
                    fc_mma(sc[j + 1], a, b[2], b[3]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int i = warp * 16 + g + 8 * r, key = j * 8 + 2 * t;
                const float x = key <= i ? sc[j][2 * r] * pw[max(i - key, 0)] : 0.f;
                const float y = key + 1 <= i ? sc[j][2 * r + 1] * pw[max(i - key - 1, 0)] : 0.f;
                uint32_t hi, lo;
                fc_split(x, y, hi, lo);
                *reinterpret_cast<uint32_t*>(ph + i * PS + key) = hi;
                *reinterpret_cast<uint32_t*>(pl + i * PS + key) = lo;
            }
    }
    // warp w: all 64 rows, columns v0 + 8 NT w …: first the state's share, straight from memory (each number is one warp's)
    float acc[4][NT][4];
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.f;
    const float* S = A.scratch + ((size_t)(start / FC + s + blockIdx.x) * A.H + h) * A.V * A.K;
    const int vw = v0 + warp * 8 * NT + g;          // this lane's column of the first tile
    auto ask = [&](int kk, float2 (&x)[NT][2]) {
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int k = kk * 16 + 2 * t + 8 * r;
                x[j][r] = (vw + 8 * j < A.V && k < A.K) ? *reinterpret_cast<const float2*>(S + (size_t)(vw + 8 * j) * A.K + k) : make_float2(0.f, 0.f);
            }
    };
    float2 now[NT][2], next[NT][2];
    ask(0, now);
    for (int kk = 0; kk < K16 / 16; ++kk) {
        if (kk + 1 < K16 / 16) ask(kk + 1, next);
        uint32_t bh[NT][2], bl[NT][2];
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int r = 0; r < 2; ++r) fc_split(now[j][r].x, now[j][r].y, bh[j][r], bl[j][r]);
#pragma unroll
        for (int m = 0; m < 4; ++m) {
            uint32_t a[4];
            fc_ldsm(a, fc_sm(qs + (m * 16 + (lane & 15)) * KS + kk * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                fc_mma(acc[m][j], a, bh[j][0], bh[j][1]);
                fc_mma(acc[m][j], a, bl[j][0], bl[j][1]);
            }
        }
#pragma unroll
        for (int j = 0; j < NT; ++j) { now[j][0] = next[j][0]; now[j][1] = next[j][1]; }
    }
#pragma unroll
    for (int m = 0; m < 4; ++m) {
        const float f0 = pw[m * 16 + g + 1], f1 = pw[m * 16 + g + 9];
#pragma unroll
        for (int j = 0; j < NT; ++j) { acc[m][j][0] *= f0; acc[m][j][1] *= f0; acc[m][j][2] *= f1; acc[m][j][3] *= f1; }
    }
    __syncthreads();                                // every warp's scores are there
#pragma unroll
    for (int kk = 0; kk < FC / 16; ++kk) {
        uint32_t b[NT][2];
#pragma unroll
        for (int j = 0; j < NT; ++j) fc_ldsm_t2(b[j][0], b[j][1], fc_sm(vs + (kk * 16 + (lane & 15)) * VS + (warp * NT + j) * 8));
#pragma unroll
        for (int m = kk; m < 4; ++m) {              // (tokens 16 kk … are behind the rows of the tiles before)
            uint32_t a[4];
            fc_ldsm(a, fc_sm(ph + (m * 16 + (lane & 15)) * PS + kk * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int j = 0; j < NT; ++j) fc_mma(acc[m][j], a, b[j][0], b[j][1]);
            fc_ldsm(a, fc_sm(pl + (m * 16 + (lane & 15)) * PS + kk * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int j = 0; j < NT; ++j) fc_mma(acc[m][j], a, b[j][0], b[j][1]);
        }
    }
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int i = m * 16 + g + 8 * r;
            if (i >= L) continue;
            float* dst = A.y + (size_t)(start + c0 + i) * A.ldy + (size_t)h * A.V;
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int v = v0 + (warp * NT + j) * 8 + 2 * t;
                if (v < A.V) *reinterpret_cast<float2*>(dst + v) = make_float2(acc[m][j][2 * r] * A.q_scale, acc[m][j][2 * r + 1] * A.q_scale);
            }
        }
}

template <int NT> int launch_outputs(const FixedChunks& A, int chunks, int n_seqs, cudaStream_t stream) {
    constexpr int VT = 32 * NT;
    const int KS = ((A.K + 15) & ~15) + 8, v_tiles = (A.V + VT - 1) / VT;
    const size_t smem = (size_t)(2 * FC * KS + FC * (VT + 8) + 2 * FC * (FC + 8)) * 2 + (FC + 1) * 4;
    static size_t allowed = 48 * 1024;
    if (smem > allowed) {
        const cudaError_t e = cudaFuncSetAttribute(chunk_outputs_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return vlrf_fail(VLRF_ERR_CUDA, "fixed_state_chunks: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        allowed = smem;
    }
    launch_chained(chunk_outputs_kernel<NT>, dim3(chunks, A.H * v_tiles, n_seqs), dim3(128), smem, stream, A, v_tiles);
    return vlrf_check_launch("fixed_state_chunks: outputs");
}
}  // namespace

// Whether the chunked kernels take these sizes: state rows up to 256 and columns, both multiples of 8 (rows on 16-byte boundaries).
extern "C" int vlrf_fixed_state_chunks_takes(int K, int V, int ldq, int ldk, int ldv, int ldy, int state_row) {
    return (K > 0 && K <= FC_MAX_K && K % 8 == 0 && V > 0 && V <= 4096 && V % 8 == 0 && ldq % 8 == 0 && ldk % 8 == 0 && ldv % 8 == 0 && ldy % 2 == 0 &&
            state_row % 4 == 0) ? 1 : 0;
}

// float32 scratch of a step of T tokens in n_seqs sequences
extern "C" long long vlrf_fixed_state_chunks_scratch(int T, int n_seqs, int H, int K, int V) {
    return ((long long)T / FC + n_seqs) * H * K * V;
}

extern "C" int vlrf_fixed_state_chunks(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, const float* decay, float q_scale,
                                       float* scratch, float* state, int state_row, const int* seq_slot, const int* seq_start, const int* seq_pos0,
                                       float* y, int ldy, int n_seqs, int max_new, int H, int K, int V, cudaStream_t stream) {
    VLRF_REQUIRE(vlrf_fixed_state_chunks_takes(K, V, ldq, ldk, ldv, ldy, state_row), "fixed_state_chunks: a state of %d by %d or the rows' strides are not taken", K, V);
    VLRF_REQUIRE(n_seqs >= 0 && max_new >= 0 && H > 0 && n_seqs <= 65535 && decay != nullptr && scratch != nullptr, "fixed_state_chunks: bad arguments");
    VLRF_REQUIRE(ldq >= H * K && ldk >= H * K && ldv >= H * V && ldy >= H * V && (long long)H * K * V <= state_row, "fixed_state_chunks: columns lie outside the rows");
    VLRF_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(state) |
                   reinterpret_cast<uintptr_t>(scratch)) & 15) == 0 && (reinterpret_cast<uintptr_t>(y) & 7) == 0, "fixed_state_chunks: misaligned rows");
    if (n_seqs == 0 || max_new == 0) return VLRF_OK;
    const int chunks = (max_new + FC - 1) / FC, k_tiles = (K + 63) / 64, v_tiles = (V + 63) / 64;
    VLRF_REQUIRE((long long)H * k_tiles * v_tiles <= 65535, "fixed_state_chunks: too many heads");
    const FixedChunks A{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, ldq, ldk, ldv, decay, q_scale, scratch, state, y,
                        state_row, ldy, seq_slot, seq_start, seq_pos0, H, K, V};
    launch_chained(chunk_writes_kernel, dim3(chunks, H * k_tiles * v_tiles, n_seqs), dim3(128), (size_t)0, stream, A, k_tiles, v_tiles);
    int st = vlrf_check_launch("fixed_state_chunks: writes");
    if (st != VLRF_OK) return st;
    const long long quads = (long long)H * K * V / 4;
    launch_chained(chunk_states_kernel, dim3((unsigned)((quads + 127) / 128), n_seqs), dim3(128), (size_t)0, stream, A);
    st = vlrf_check_launch("fixed_state_chunks: states");
    if (st != VLRF_OK) return st;
    if (V <= 32) return launch_outputs<1>(A, chunks, n_seqs, stream);
    if (V <= 64) return launch_outputs<2>(A, chunks, n_seqs, stream);
    return launch_outputs<4>(A, chunks, n_seqs, stream);
}
