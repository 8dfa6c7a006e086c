// The row-wise kernels around the recurrences of matrix_state.cu.
//
// conv_unit: queries, keys and values of a recurrence from the float32 rows of a layer's input product, which hold
//   [q: G·K | k: G·K | v: H·V] from x_off on: a causal convolution per channel (taps − 1 earlier inputs: rows of this step
//   or the sequence's kept inputs; the last tap is the current token's; no bias), x · sigmoid(x), and for q and k the
//   division by sqrt(Σ x² + 1e-6) over the head.  Also leaves k · q per head (`kq` [T][G]) and the last taps − 1 inputs of
//   every sequence: they follow the states in the sequence's state row (see matrix_state.cu for its two copies), at
//   conv_off, [taps − 1][channels].  A warp takes a head (a query head with its key head, or a value head) and a run of
//   tokens: the head's channels in registers, a run's inputs read once.
// lowrank_rows: out[t][c] = f(Σ_r a[t][r] · w[c][r] + bias[c]), a short product behind a short product, in float32 from the
//   float32 rows a (bfloat16 weights: the rows are split into two bfloat16 halves and multiplied by `mma.sync`, float32
//   weights: multiply-adds).  f: nothing; sigmoid(z)^(1/tau) (a decay); exp(−exp(a_log[c / per]) · softplus(z)) (a decay).
//   Two such products, each with its own rows, weights and f, run in one launch.
// head_rows: out[t][h·V + i] = factor · o / sqrt(mean(o²) + eps) · w · act(gate[t][h·V + i]) with the mean over the head's V
//   numbers; o = y, or y / (max(|n·q|, floor) + 1e-6) where `den` gives (n·q, floor) per token and head; w one vector of V
//   numbers for all heads or of H·V numbers; act sigmoid(z) or z · sigmoid(z); rounded to the activation dtype.  A warp per token
//   and head, or, where heads are wide (all heads of a mixer normed as one row, H = 1), a CTA.
// norm_pair_add: x[t] += factor · (RMSnorm(a[t]) · wa + RMSnorm(b[t]) · wb), float32; the rows fit registers.
#include "common.cuh"
#include <type_traits>

namespace {
constexpr float UNIT_EPS = 1e-6f, DEN_EPS = 1e-6f;

// ---- convolution, unit norms -----------------------------------------------------------------------------------------
// CPL: channels a lane (a head of up to 32·CPL); R: tokens a run; TAPS: taps known at compile time, or 0
template <int CPL, int R, int TAPS>
__global__ void __launch_bounds__(128)
conv_unit_kernel(const float* __restrict__ proj, int ld, int x_off, const float* __restrict__ w, int taps_rt, float* __restrict__ state,
                 int state_row, int conv_off, const int* __restrict__ seq_slot, const int* __restrict__ seq_start,
                 const int* __restrict__ seq_pos0, float* __restrict__ out, float* __restrict__ kq, int H, int G, int K, int V, int channels,
                 int keep_here) {
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.x * 4 + warp, s = blockIdx.y;
    if (unit >= G + H) return;                      // (whole warps; no block-wide barrier below)
    const int slot = seq_slot[s];
    if (slot < 0) return;
    const int start = seq_start[s], n = seq_start[s + 1] - start, pos0 = seq_pos0[s];
    const int i0 = blockIdx.z * R;
    if (i0 >= n) return;
    const int i1 = min(n, i0 + R);
    const int taps = TAPS ? TAPS : taps_rt;
    const float* kept = state + ((size_t)slot * 2 + (pos0 & 1)) * state_row + conv_off;
    float* next = state + ((size_t)slot * 2 + ((pos0 + n) & 1)) * state_row + conv_off;
    // the input of channel c at place i of the step (negative: a kept input)
    auto input = [&](int i, int c) -> float {
        return i >= 0 ? proj[(size_t)(start + i) * ld + x_off + c] : kept[(size_t)(taps - 1 + i) * channels + c];
    };
    float val[CPL][R];
    auto convolve = [&](int c0, int len) {          // channels c0 + lane + 32 j
#pragma unroll
        for (int j = 0; j < CPL; ++j) {
            const int cc = lane + 32 * j;
#pragma unroll
            for (int t = 0; t < R; ++t) val[j][t] = 0.f;
            if (cc < len) {
                const int ch = c0 + cc;
                if (TAPS) {
                    float in[R + (TAPS ? TAPS - 1 : 0)], wt[TAPS ? TAPS : 1];
#pragma unroll
                    for (int q = 0; q < TAPS; ++q) wt[q] = w[(size_t)ch * TAPS + q];
#pragma unroll
                    for (int q = 0; q < R + TAPS - 1; ++q) {
                        const int i = i0 + q - (TAPS - 1);
                        in[q] = i < i1 ? input(i, ch) : 0.f;
                    }
#pragma unroll
                    for (int t = 0; t < R; ++t) {
                        float a = 0.f;
#pragma unroll
                        for (int q = 0; q < TAPS; ++q) a = fmaf(wt[q], in[t + q], a);
                        val[j][t] = silu_f(a);
                    }
                } else {
#pragma unroll
                    for (int t = 0; t < R; ++t) {
                        if (i0 + t < i1) {
                            float a = 0.f;
                            for (int q = 0; q < taps; ++q) a = fmaf(w[(size_t)ch * taps + q], input(i0 + t - (taps - 1) + q, ch), a);
                            val[j][t] = silu_f(a);
                        }
                    }
                }
            }
        }
    };
    auto keep_inputs = [&](int c0, int len) {       // the head's last taps − 1 inputs: asked for together, then written
        if (!keep_here || i0 != 0 || taps < 2) return;
        for (int cc = lane; cc < len; cc += 32) {
            const int ch = c0 + cc;
            float in[15];
#pragma unroll
            for (int q = 0; q < (TAPS ? TAPS - 1 : 15); ++q)
                if (q < taps - 1) in[q] = input(n - (taps - 1) + q, ch);
#pragma unroll
            for (int q = 0; q < (TAPS ? TAPS - 1 : 15); ++q)
                if (q < taps - 1) next[(size_t)q * channels + ch] = in[q];
        }
    };
    auto store = [&](int c0, int len) {
#pragma unroll
        for (int t = 0; t < R; ++t) {
            if (i0 + t >= i1) break;
            float* o = out + (size_t)(start + i0 + t) * channels + c0;
#pragma unroll
            for (int j = 0; j < CPL; ++j)
                if (lane + 32 * j < len) o[lane + 32 * j] = val[j][t];
        }
    };
    if (unit >= G) {                                // a value head
        const int c0 = 2 * G * K + (unit - G) * V;
        convolve(c0, V);
        store(c0, V);
        keep_inputs(c0, V);
        return;
    }
    auto to_unit = [&]() {
#pragma unroll
        for (int t = 0; t < R; ++t) {
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < CPL; ++j) ss = fmaf(val[j][t], val[j][t], ss);
            const float inv = 1.f / sqrtf(warp_sum(ss) + UNIT_EPS);
#pragma unroll
            for (int j = 0; j < CPL; ++j) val[j][t] *= inv;
        }
    };
    const int qc = unit * K, kc = G * K + unit * K;
    convolve(qc, K);
    to_unit();
    store(qc, K);
    float qv[CPL][R];
#pragma unroll
    for (int j = 0; j < CPL; ++j)
#pragma unroll
        for (int t = 0; t < R; ++t) qv[j][t] = val[j][t];
    convolve(kc, K);
    to_unit();
    store(kc, K);
#pragma unroll
    for (int t = 0; t < R; ++t) {
        float d = 0.f;
#pragma unroll
        for (int j = 0; j < CPL; ++j) d = fmaf(qv[j][t], val[j][t], d);
        d = warp_sum(d);
        if (lane == 0 && i0 + t < i1) kq[(size_t)(start + i0 + t) * G + unit] = d;
    }
    keep_inputs(qc, K);
    keep_inputs(kc, K);
}

// The kept inputs by a launch of its own, where runs are shorter than the taps reach back (another warp's reads of the
// kept inputs must be over before they are replaced).
__global__ void __launch_bounds__(128)
conv_keep_kernel(const float* __restrict__ proj, int ld, int x_off, float* __restrict__ state, int state_row, int conv_off,
                 const int* __restrict__ seq_slot, const int* __restrict__ seq_start, const int* __restrict__ seq_pos0, int channels, int taps) {
    pdl_wait();
    pdl_launch_dependents();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
    const int slot = seq_slot[s];
    if (c >= channels || slot < 0) return;
    const int start = seq_start[s], n = seq_start[s + 1] - start, pos0 = seq_pos0[s];
    const float* kept = state + ((size_t)slot * 2 + (pos0 & 1)) * state_row + conv_off;
    float* next = state + ((size_t)slot * 2 + ((pos0 + n) & 1)) * state_row + conv_off;
    float v[15];
#pragma unroll
    for (int q = 0; q < 15; ++q) {
        if (q < taps - 1) {
            const int i = n - (taps - 1) + q;
            v[q] = i >= 0 ? proj[(size_t)(start + i) * ld + x_off + c] : kept[(size_t)(taps - 1 + i) * channels + c];
        }
    }
#pragma unroll
    for (int q = 0; q < 15; ++q)
        if (q < taps - 1) next[(size_t)q * channels + c] = v[q];
}

// ---- short products behind short products -----------------------------------------------------------------------------
constexpr int LR_PLAIN = 0, LR_POWER = 1, LR_SOFTPLUS = 2;

struct LowRankPart {
    const float* a; int lda, rank;
    const void* w;
    const float *bias, *a_log;
    int kind; float inv_tau; int per;
    float* out; int ldo, cols, tiles;
};

__device__ __forceinline__ float lr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// What f needs of a column: its bias, and for the softplus decay minus its rate.
__device__ __forceinline__ float2 lr_column(const LowRankPart& P, int col) {
    const bool in = col < P.cols;
    return make_float2(in && P.bias != nullptr ? P.bias[col] : 0.f, in && P.kind == LR_SOFTPLUS ? -expf(P.a_log[col / P.per]) : P.inv_tau);
}
template <int KIND> __device__ __forceinline__ float lr_apply(float z, float2 c) {
    z += c.x;
    if (KIND == LR_POWER) return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * c.y);      // log sigmoid(z) / tau
    if (KIND == LR_SOFTPLUS) return expf(c.y * lr_softplus(z));
    return z;
}

// a tile of 64 tokens by CT columns; bfloat16 weights on mma.sync with the float32 rows as the sum of two bfloat16 rows.  VEC: ranks
// of a multiple of 8 and rows on 16-byte boundaries, eight weights and four row entries a load
constexpr int LR_K = 64;                            // of the rank at a time
template <int CT, bool VEC>
__global__ void __launch_bounds__(128)
lowrank_mma_kernel(const LowRankPart P0, const LowRankPart P1, int T) {
    pdl_wait();
    pdl_launch_dependents();
    const bool second = (int)blockIdx.x >= P0.tiles;
    const LowRankPart P = second ? P1 : P0;
    const int c0 = (blockIdx.x - (second ? P0.tiles : 0)) * CT, t0 = blockIdx.y * 64;
    constexpr int LD = LR_K + 8;                    // rows padded against bank conflicts
    __shared__ __align__(16) __nv_bfloat16 hi[64 * LD], lo[64 * LD], ws[CT * LD];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int rank = P.rank, lda = P.lda, cols = P.cols;
    float acc[CT / 8][4];
#pragma unroll
    for (int j = 0; j < CT / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const __nv_bfloat16* W = (const __nv_bfloat16*)P.w;
    for (int r0 = 0; r0 < rank; r0 += LR_K) {
        if (r0 > 0) __syncthreads();
        const int kn = min(LR_K, (rank - r0 + 15) & ~15);       // entries that the products of this pass read
        if (VEC) {
            float4 x[64 * LR_K / 4 / 128];
            uint4 y[CT * LR_K / 8 / 128];
#pragma unroll
            for (int q = 0; q < CT * LR_K / 8 / 128; ++q) {
                const int i = threadIdx.x + q * 128, row = i / (LR_K / 8), rr = (i % (LR_K / 8)) * 8;
                y[q] = (r0 + rr < rank && c0 + row < cols) ? *reinterpret_cast<const uint4*>(W + (size_t)(c0 + row) * rank + r0 + rr) : make_uint4(0, 0, 0, 0);
            }
#pragma unroll
            for (int q = 0; q < 64 * LR_K / 4 / 128; ++q) {
                const int i = threadIdx.x + q * 128, row = i / (LR_K / 4), rr = (i % (LR_K / 4)) * 4;
                x[q] = (r0 + rr < rank && t0 + row < T) ? *reinterpret_cast<const float4*>(P.a + (size_t)(t0 + row) * lda + r0 + rr) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int q = 0; q < CT * LR_K / 8 / 128; ++q) {
                const int i = threadIdx.x + q * 128, row = i / (LR_K / 8), rr = (i % (LR_K / 8)) * 8;
                *reinterpret_cast<uint4*>(ws + row * LD + rr) = y[q];
            }
#pragma unroll
            for (int q = 0; q < 64 * LR_K / 4 / 128; ++q) {
                const int i = threadIdx.x + q * 128, row = i / (LR_K / 4), rr = (i % (LR_K / 4)) * 4;
                const __nv_bfloat162 h0 = __floats2bfloat162_rn(x[q].x, x[q].y), h1 = __floats2bfloat162_rn(x[q].z, x[q].w);
                const __nv_bfloat162 l0 = __floats2bfloat162_rn(x[q].x - __low2float(h0), x[q].y - __high2float(h0));
                const __nv_bfloat162 l1 = __floats2bfloat162_rn(x[q].z - __low2float(h1), x[q].w - __high2float(h1));
                *reinterpret_cast<uint2*>(hi + row * LD + rr) = make_uint2(*reinterpret_cast<const uint32_t*>(&h0), *reinterpret_cast<const uint32_t*>(&h1));
                *reinterpret_cast<uint2*>(lo + row * LD + rr) = make_uint2(*reinterpret_cast<const uint32_t*>(&l0), *reinterpret_cast<const uint32_t*>(&l1));
            }
        } else {
            for (int i = threadIdx.x; i < 64 * kn; i += 128) {
                const int row = i / kn, rr = i - row * kn;
                const float x = (r0 + rr < rank && t0 + row < T) ? P.a[(size_t)(t0 + row) * lda + r0 + rr] : 0.f;
                const __nv_bfloat16 h = __float2bfloat16_rn(x);
                hi[row * LD + rr] = h;
                lo[row * LD + rr] = __float2bfloat16_rn(x - __bfloat162float(h));
                if (row < CT) ws[row * LD + rr] = (r0 + rr < rank && c0 + row < cols) ? W[(size_t)(c0 + row) * rank + r0 + rr] : __float2bfloat16_rn(0.f);
            }
        }
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < LR_K / 16; ++ks) {
            if (16 * ks >= kn) break;
            uint32_t ah[4], al[4];
            const int rb = warp * 16 + g, kb = ks * 16 + 2 * t;
#pragma unroll
            for (int q = 0; q < 4; ++q) {           // (row g or g + 8; k low or high half)
                const int at = (rb + (q & 1) * 8) * LD + kb + (q >> 1) * 8;
                ah[q] = *reinterpret_cast<const uint32_t*>(hi + at);
                al[q] = *reinterpret_cast<const uint32_t*>(lo + at);
            }
#pragma unroll
            for (int j = 0; j < CT / 8; ++j) {
                const uint32_t b0 = *reinterpret_cast<const uint32_t*>(ws + (j * 8 + g) * LD + kb);
                const uint32_t b1 = *reinterpret_cast<const uint32_t*>(ws + (j * 8 + g) * LD + kb + 8);
#define LR_MMA(A) asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n" \
                               : "+f"(acc[j][0]), "+f"(acc[j][1]), "+f"(acc[j][2]), "+f"(acc[j][3]) \
                               : "r"(A[0]), "r"(A[1]), "r"(A[2]), "r"(A[3]), "r"(b0), "r"(b1))
                LR_MMA(al);
                LR_MMA(ah);
#undef LR_MMA
            }
        }
    }
    float* out = P.out;
    const int ldo = P.ldo;
    const bool pairs = (ldo & 1) == 0 && (cols & 1) == 0 && (reinterpret_cast<uintptr_t>(out) & 7) == 0;
    auto finish = [&](auto kind) {
        constexpr int KIND = decltype(kind)::value;
#pragma unroll
        for (int j = 0; j < CT / 8; ++j) {
            const int col = c0 + j * 8 + 2 * t;
            if (col >= cols) break;
            const float2 k0 = lr_column(P, col), k1 = lr_column(P, col + 1);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int row = t0 + warp * 16 + g + half * 8;
                if (row >= T) continue;
                float* o = out + (size_t)row * ldo + col;
                const float x0 = lr_apply<KIND>(acc[j][2 * half], k0), x1 = lr_apply<KIND>(acc[j][2 * half + 1], k1);
                if (pairs) *reinterpret_cast<float2*>(o) = make_float2(x0, x1);
                else {
                    o[0] = x0;
                    if (col + 1 < cols) o[1] = x1;
                }
            }
        }
    };
    if (P.kind == LR_SOFTPLUS) finish(std::integral_constant<int, LR_SOFTPLUS>{});
    else if (P.kind == LR_POWER) finish(std::integral_constant<int, LR_POWER>{});
    else finish(std::integral_constant<int, LR_PLAIN>{});
}

// float32 weights: the same tile, four by eight results a thread
__global__ void __launch_bounds__(128)
lowrank_fma_kernel(const LowRankPart P0, const LowRankPart P1, int T) {
    pdl_wait();
    pdl_launch_dependents();
    const bool second = (int)blockIdx.x >= P0.tiles;
    const LowRankPart& P = second ? P1 : P0;
    const int c0 = (blockIdx.x - (second ? P0.tiles : 0)) * 64, t0 = blockIdx.y * 64;
    __shared__ float as[16][65], ws[16][65];
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const float* W = (const float*)P.w;
    for (int r0 = 0; r0 < P.rank; r0 += 16) {
        if (r0 > 0) __syncthreads();
        for (int i = threadIdx.x; i < 64 * 16; i += 128) {
            const int row = i >> 4, rr = i & 15;
            const bool in = r0 + rr < P.rank;
            as[rr][row] = (in && t0 + row < T) ? P.a[(size_t)(t0 + row) * P.lda + r0 + rr] : 0.f;
            ws[rr][row] = (in && c0 + row < P.cols) ? W[(size_t)(c0 + row) * P.rank + r0 + rr] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int rr = 0; rr < 16; ++rr)
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(as[rr][ty + 8 * i], ws[rr][tx + 16 * j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int row = t0 + ty + 8 * i;
        if (row >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int col = c0 + tx + 16 * j;
            if (col >= P.cols) continue;
            const float2 c = lr_column(P, col);
            P.out[(size_t)row * P.ldo + col] = P.kind == LR_SOFTPLUS ? lr_apply<LR_SOFTPLUS>(acc[i][j], c)
                                               : P.kind == LR_POWER ? lr_apply<LR_POWER>(acc[i][j], c) : lr_apply<LR_PLAIN>(acc[i][j], c);
        }
    }
}

// ---- a head's read-out ------------------------------------------------------------------------------------------------
template <typename OT> __device__ __forceinline__ void store4(OT* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store4<float>(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
    const __nv_bfloat162 l = __floats2bfloat162_rn(a, b), h = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&l), *reinterpret_cast<const uint32_t*>(&h));
}

// a warp per (token, head).  VEC: heads of a multiple of 4 up to 128·4, everything on 16-byte boundaries, four numbers a lane
template <typename OT, bool VEC>
__global__ void __launch_bounds__(128)
head_rows_kernel(const float* __restrict__ y, int ldy, const float* __restrict__ den, const float* __restrict__ w, int w_per_head,
                 const float* __restrict__ gate, int ld_gate, int act, OT* __restrict__ out, int ld_out, int T, int H, int V, float eps, float factor) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const long long at = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (at >= (long long)T * H) return;             // (whole warps)
    const int t = (int)(at / H), h = (int)(at - (long long)t * H);
    const float* yr = y + (size_t)t * ldy + (size_t)h * V;
    const float* gr = gate + (size_t)t * ld_gate + (size_t)h * V;
    const float* wr = w + (w_per_head ? (size_t)h * V : 0);
    OT* o = out + (size_t)t * ld_out + (size_t)h * V;
    float inv_den = 1.f;
    if (den != nullptr) {
        const float2 d = *reinterpret_cast<const float2*>(den + (size_t)at * 2);
        inv_den = 1.f / (fmaxf(fabsf(d.x), d.y) + DEN_EPS);
    }
    auto gated = [&](float z) { return act == VLRF_ACT_SILU ? silu_f(z) : sigmoid_f(z); };
    float ss = 0.f;
    if (VEC) {
        float4 v[4], gt[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = 4 * (lane + 32 * j);
            v[j] = gt[j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < V) { v[j] = *reinterpret_cast<const float4*>(yr + i); gt[j] = *reinterpret_cast<const float4*>(gr + i); }
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            v[j].x *= inv_den; v[j].y *= inv_den; v[j].z *= inv_den; v[j].w *= inv_den;
            ss = fmaf(v[j].x, v[j].x, ss); ss = fmaf(v[j].y, v[j].y, ss); ss = fmaf(v[j].z, v[j].z, ss); ss = fmaf(v[j].w, v[j].w, ss);
        }
        const float inv = factor / sqrtf(warp_sum(ss) / (float)V + eps);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = 4 * (lane + 32 * j);
            if (i < V) {
                const float4 ww = *reinterpret_cast<const float4*>(wr + i);
                store4<OT>(o + i, v[j].x * inv * ww.x * gated(gt[j].x), v[j].y * inv * ww.y * gated(gt[j].y),
                           v[j].z * inv * ww.z * gated(gt[j].z), v[j].w * inv * ww.w * gated(gt[j].w));
            }
        }
    } else {
        for (int i = lane; i < V; i += 32) { const float v = yr[i] * inv_den; ss = fmaf(v, v, ss); }
        const float inv = factor / sqrtf(warp_sum(ss) / (float)V + eps);
        for (int i = lane; i < V; i += 32) ElemIO<OT>::store(o + i, yr[i] * inv_den * inv * wr[i] * gated(gr[i]));
    }
}

// A CTA per (token, head) for wide heads.  NV: quads of columns a thread holds in registers (rows on 16-byte boundaries, V a
// multiple of 4 up to 1024·NV); 0: any sizes, a column at a time.
template <typename OT, int NV>
__global__ void __launch_bounds__(256)
head_rows_wide_kernel(const float* __restrict__ y, int ldy, const float* __restrict__ den, const float* __restrict__ w, int w_per_head,
                      const float* __restrict__ gate, int ld_gate, int act, OT* __restrict__ out, int ld_out, int H, int V, float eps, float factor) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float red[8];
    const int t = blockIdx.x / H, h = blockIdx.x - t * H, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* yr = y + (size_t)t * ldy + (size_t)h * V;
    const float* gr = gate + (size_t)t * ld_gate + (size_t)h * V;
    const float* wr = w + (w_per_head ? (size_t)h * V : 0);
    OT* o = out + (size_t)t * ld_out + (size_t)h * V;
    float inv_den = 1.f;
    if (den != nullptr) {
        const float2 d = *reinterpret_cast<const float2*>(den + (size_t)blockIdx.x * 2);
        inv_den = 1.f / (fmaxf(fabsf(d.x), d.y) + DEN_EPS);
    }
    auto gated = [&](float z) { return act == VLRF_ACT_SILU ? silu_f(z) : sigmoid_f(z); };
    auto all = [&](float ss) -> float {             // the sum over the CTA
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        return ((red[0] + red[1]) + (red[2] + red[3])) + ((red[4] + red[5]) + (red[6] + red[7]));
    };
    float ss = 0.f;
    if constexpr (NV > 0) {
        float4 v[NV], gt[NV];
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = 4 * (threadIdx.x + 256 * k);
            v[k] = gt[k] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i < V) { v[k] = *reinterpret_cast<const float4*>(yr + i); gt[k] = *reinterpret_cast<const float4*>(gr + i); }
        }
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            v[k].x *= inv_den; v[k].y *= inv_den; v[k].z *= inv_den; v[k].w *= inv_den;
            ss = fmaf(v[k].x, v[k].x, ss); ss = fmaf(v[k].y, v[k].y, ss); ss = fmaf(v[k].z, v[k].z, ss); ss = fmaf(v[k].w, v[k].w, ss);
        }
        const float inv = factor / sqrtf(all(ss) / (float)V + eps);
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int i = 4 * (threadIdx.x + 256 * k);
            if (i < V) {
                const float4 ww = *reinterpret_cast<const float4*>(wr + i);
                store4<OT>(o + i, v[k].x * inv * ww.x * gated(gt[k].x), v[k].y * inv * ww.y * gated(gt[k].y),
                           v[k].z * inv * ww.z * gated(gt[k].z), v[k].w * inv * ww.w * gated(gt[k].w));
            }
        }
    } else {
        for (int i = threadIdx.x; i < V; i += 256) { const float v = yr[i] * inv_den; ss = fmaf(v, v, ss); }
        const float inv = factor / sqrtf(all(ss) / (float)V + eps);
        for (int i = threadIdx.x; i < V; i += 256) ElemIO<OT>::store(o + i, yr[i] * inv_den * inv * wr[i] * gated(gr[i]));
    }
}

// ---- two normed rows added to the residual ------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
norm_pair_add_kernel(const float* __restrict__ a, const float* __restrict__ b, const float* __restrict__ wa, const float* __restrict__ wb,
                     float* __restrict__ x, int d, float eps, float factor, int accumulate) {
    pdl_wait();
    pdl_launch_dependents();
    __shared__ float red[2][8];
    const size_t at = (size_t)blockIdx.x * d;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x; i < d; i += 256) { sa = fmaf(a[at + i], a[at + i], sa); sb = fmaf(b[at + i], b[at + i], sb); }
    sa = warp_sum(sa);
    sb = warp_sum(sb);
    if (lane == 0) { red[0][warp] = sa; red[1][warp] = sb; }
    __syncthreads();
    sa = sb = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) { sa += red[0][i]; sb += red[1][i]; }
    const float ia = factor / sqrtf(sa / (float)d + eps), ib = factor / sqrtf(sb / (float)d + eps);
    for (int i = threadIdx.x; i < d; i += 256) {
        const float v = a[at + i] * ia * wa[i] + b[at + i] * ib * wb[i];
        x[at + i] = accumulate ? x[at + i] + v : v;
    }
}

bool rows16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <int CPL, int R, int TAPS>
void launch_conv(const float* proj, int ld, int x_off, const float* w, int taps, float* state, int state_row, int conv_off,
                 const int* seq_slot, const int* seq_start, const int* seq_pos0, float* out, float* kq, int n_seqs, int max_new, int H, int G,
                 int K, int V, int channels, cudaStream_t stream) {
    // the warp of a run that reads kept inputs also replaces them, unless several runs read them
    const int keep_here = (taps - 1 <= R || max_new <= R) ? 1 : 0;
    launch_chained(conv_unit_kernel<CPL, R, TAPS>, dim3((G + H + 3) / 4, n_seqs, (max_new + R - 1) / R), dim3(128), (size_t)0, stream, proj, ld,
                   x_off, w, taps, state, state_row, conv_off, seq_slot, seq_start, seq_pos0, out, kq, H, G, K, V, channels, keep_here);
    if (!keep_here)
        launch_chained(conv_keep_kernel, dim3((channels + 127) / 128, n_seqs), dim3(128), (size_t)0, stream, proj, ld, x_off, state, state_row,
                       conv_off, seq_slot, seq_start, seq_pos0, channels, taps);
}
}  // namespace

extern "C" int vlrf_conv_unit(const float* proj, int ld, int x_off, const float* w, int taps, float* state, int state_row, int conv_off,
                              const int* seq_slot, const int* seq_start, const int* seq_pos0, float* out, float* kq, int n_seqs, int max_new,
                              int H, int G, int K, int V, cudaStream_t stream) {
    VLRF_REQUIRE(n_seqs >= 0 && max_new >= 0 && H > 0 && G > 0 && K > 0 && V > 0, "conv_unit: bad sizes");
    VLRF_REQUIRE(taps >= 1 && taps <= 16, "conv_unit: %d taps are not in 1…16", taps);
    VLRF_REQUIRE(K <= 512 && V <= 512 && n_seqs <= 65535, "conv_unit: heads of %d and %d channels are above 512, or too many sequences", K, V);
    const int channels = 2 * G * K + H * V;
    VLRF_REQUIRE(x_off >= 0 && x_off + channels <= ld && (long long)conv_off + (long long)(taps - 1) * channels <= state_row, "conv_unit: columns lie outside the row");
    if (n_seqs == 0 || max_new == 0) return VLRF_OK;
    const int widest = K > V ? K : V;
#define ARGS proj, ld, x_off, w, taps, state, state_row, conv_off, seq_slot, seq_start, seq_pos0, out, kq, n_seqs, max_new, H, G, K, V, channels, stream
#define GO(CPL, R) do { if (taps == 4) launch_conv<CPL, R, 4>(ARGS); else launch_conv<CPL, R, 0>(ARGS); } while (0)
    const bool single = max_new == 1;
    if (widest <= 32) { if (single) GO(1, 1); else GO(1, 8); }
    else if (widest <= 64) { if (single) GO(2, 1); else GO(2, 8); }
    else if (widest <= 128) { if (single) GO(4, 1); else GO(4, 4); }
    else if (widest <= 256) { if (single) GO(8, 1); else GO(8, 4); }
    else { if (single) GO(16, 1); else GO(16, 2); }
#undef GO
#undef ARGS
    return vlrf_check_launch("conv_unit");
}

static int lowrank_part(LowRankPart& P, const float* a, int lda, int rank, const void* w, const float* bias, const float* a_log, int kind,
                        float tau, int per, float* out, int ldo, int cols) {
    VLRF_REQUIRE(a != nullptr && w != nullptr && out != nullptr && rank > 0 && cols > 0 && lda >= rank && ldo >= cols, "lowrank_rows: bad sizes");
    VLRF_REQUIRE(kind >= LR_PLAIN && kind <= LR_SOFTPLUS && (kind != LR_POWER || tau > 0.f) && (kind != LR_SOFTPLUS || (a_log != nullptr && per > 0)),
                 "lowrank_rows: unknown function %d, or its constants are missing", kind);
    P.a = a; P.lda = lda; P.rank = rank; P.w = w; P.bias = bias; P.a_log = a_log; P.kind = kind;
    P.inv_tau = kind == LR_POWER ? 1.f / tau : 1.f; P.per = per > 0 ? per : 1; P.out = out; P.ldo = ldo; P.cols = cols; P.tiles = (cols + 63) / 64;
    return VLRF_OK;
}

extern "C" int vlrf_lowrank_rows(const float* a0, int lda0, int rank0, const void* w0, const float* bias0, const float* a_log0, int kind0, float tau0,
                                 int per0, float* out0, int ldo0, int cols0, const float* a1, int lda1, int rank1, const void* w1,
                                 const float* bias1, const float* a_log1, int kind1, float tau1, int per1, float* out1, int ldo1, int cols1,
                                 int w_dtype, int T, cudaStream_t stream) {
    LowRankPart P0, P1;
    int st = lowrank_part(P0, a0, lda0, rank0, w0, bias0, a_log0, kind0, tau0, per0, out0, ldo0, cols0);
    if (st != VLRF_OK) return st;
    P1 = P0;
    P1.tiles = 0;
    if (a1 != nullptr) {
        st = lowrank_part(P1, a1, lda1, rank1, w1, bias1, a_log1, kind1, tau1, per1, out1, ldo1, cols1);
        if (st != VLRF_OK) return st;
    }
    VLRF_REQUIRE(T >= 0 && T <= 64 * 65535, "lowrank_rows: too many rows");
    if (T == 0) return VLRF_OK;
    const dim3 grid(P0.tiles + P1.tiles, (T + 63) / 64);
    if (w_dtype == VLRF_BF16) {
        // few rows: narrower tiles, so that more of the GPU takes part
        const int ct = T <= 64 ? 32 : 64;
        P0.tiles = (P0.cols + ct - 1) / ct;
        P1.tiles = a1 != nullptr ? (P1.cols + ct - 1) / ct : 0;
        const dim3 g(P0.tiles + P1.tiles, (T + 63) / 64);
        const auto fits = [](const LowRankPart& P) { return P.rank % 8 == 0 && P.lda % 4 == 0 && rows16(P.a) && rows16(P.w); };
        const bool vec = fits(P0) && fits(P1);
        if (ct == 32) { if (vec) launch_chained(lowrank_mma_kernel<32, true>, g, dim3(128), (size_t)0, stream, P0, P1, T);
                        else launch_chained(lowrank_mma_kernel<32, false>, g, dim3(128), (size_t)0, stream, P0, P1, T); }
        else { if (vec) launch_chained(lowrank_mma_kernel<64, true>, g, dim3(128), (size_t)0, stream, P0, P1, T);
               else launch_chained(lowrank_mma_kernel<64, false>, g, dim3(128), (size_t)0, stream, P0, P1, T); }
    }
    else if (w_dtype == VLRF_F32) launch_chained(lowrank_fma_kernel, grid, dim3(128), (size_t)0, stream, P0, P1, T);
    else return vlrf_fail(VLRF_ERR_INVALID_ARG, "lowrank_rows: unknown weight dtype %d", w_dtype);
    return vlrf_check_launch("lowrank_rows");
}

extern "C" int vlrf_head_rows(const float* y, int ldy, const float* den, const float* w, int w_per_head, const float* gate, int ld_gate, int act,
                              void* out, int out_dtype, int ld_out, int T, int H, int V, float eps, float factor, cudaStream_t stream) {
    VLRF_REQUIRE(T >= 0 && H > 0 && V > 0 && ldy >= H * V && ld_gate >= H * V && ld_out >= H * V, "head_rows: bad sizes");
    VLRF_REQUIRE(act == VLRF_ACT_SILU || act == VLRF_ACT_SIGMOID, "head_rows: the gate is sigmoid(z) or z·sigmoid(z)");
    if (T == 0) return VLRF_OK;
    const long long warps = (long long)T * H;
    VLRF_REQUIRE(warps <= 0x7fffffffLL, "head_rows: too many rows");
    const dim3 grid((unsigned)((warps + 3) / 4)), block(128);
    const int es = out_dtype == VLRF_BF16 ? 8 : 16;
    const bool quads = V % 4 == 0 && rows16(y) && ldy % 4 == 0 && rows16(gate) && ld_gate % 4 == 0 && rows16(w) &&
                     (reinterpret_cast<uintptr_t>(out) & (es - 1)) == 0 && ld_out % 4 == 0;
    if (V > 512) {                                  // wide heads: a CTA each
#define WIDE(OT, NV) launch_chained(head_rows_wide_kernel<OT, NV>, dim3((unsigned)warps), dim3(256), (size_t)0, stream, y, ldy, den, w, w_per_head, gate, ld_gate, act, (OT*)out, ld_out, H, V, eps, factor)
#define WIDE_NV(OT) do { if (!quads || V > 8192) WIDE(OT, 0); else if (V <= 1024) WIDE(OT, 1); else if (V <= 2048) WIDE(OT, 2); else if (V <= 4096) WIDE(OT, 4); else WIDE(OT, 8); } while (0)
        if (out_dtype == VLRF_F32) WIDE_NV(float);
        else if (out_dtype == VLRF_BF16) WIDE_NV(__nv_bfloat16);
        else return vlrf_fail(VLRF_ERR_INVALID_ARG, "head_rows: unknown output dtype %d", out_dtype);
#undef WIDE_NV
#undef WIDE
        return vlrf_check_launch("head_rows");
    }
    const bool vec = quads;
#define GO(OT, VEC) launch_chained(head_rows_kernel<OT, VEC>, grid, block, (size_t)0, stream, y, ldy, den, w, w_per_head, gate, ld_gate, act, (OT*)out, ld_out, T, H, V, eps, factor)
    if (out_dtype == VLRF_F32) { if (vec) GO(float, true); else GO(float, false); }
    else if (out_dtype == VLRF_BF16) { if (vec) GO(__nv_bfloat16, true); else GO(__nv_bfloat16, false); }
    else return vlrf_fail(VLRF_ERR_INVALID_ARG, "head_rows: unknown output dtype %d", out_dtype);
#undef GO
    return vlrf_check_launch("head_rows");
}

extern "C" int vlrf_norm_pair_add(const float* a, const float* b, const float* wa, const float* wb, float* x, int n_rows, int d, float eps,
                                  float factor, int accumulate, cudaStream_t stream) {
    VLRF_REQUIRE(n_rows >= 0 && d > 0, "norm_pair_add: bad sizes");
    if (n_rows == 0) return VLRF_OK;
    launch_chained(norm_pair_add_kernel, dim3(n_rows), dim3(256), (size_t)0, stream, a, b, wa, wb, x, d, eps, factor, accumulate);
    return vlrf_check_launch("norm_pair_add");
}
