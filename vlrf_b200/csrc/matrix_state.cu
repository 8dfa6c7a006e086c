// Recurrences with a matrix state per head, token by token in float32.
//
// A head keeps a matrix S of K rows (key channels) by V columns (value channels).  A token brings k and q (K numbers
// each, shared by the H / G heads of a group), v (V numbers) and what the kind of recurrence asks for:
//   kind 0, decayed      S ← diag(a) S + k vᵀ,                                        o = Sᵀ q
//                        a: a factor per head and key channel, read as it is (rows of `decay`)
//   kind 1, delta        S ← diag(a) S,  u = b (v − Sᵀ k),  S ← S + k uᵀ,             o = Sᵀ q
//                        a as above; b = sigmoid(s0), a number per head; s1 = k · q of the token, a number per group
//   kind 2, stabilized   m' = max(f + m, i),  S ← exp(f + m − m') S + exp(i − m') k vᵀ,  n ← the same with k alone
//                        with log gates i = c tanh(s0 / c), f = log sigmoid(c tanh(s1 / c)) per head; leaves Sᵀ q in y,
//                        and n · q and exp(−m') in `den` (what divides one by the other stands with the kernel that reads them)
//   kind 3, fixed        S ← a S + k vᵀ,                                              o = Sᵀ q
//                        a: one number per head, the same for every token (`decay` [H])
// In kind 3 q, k and v may be raw projections that go through x · sigmoid(x) here (`input_act`): a thread applies it to what it has
// copied into shared memory itself, ahead of the barrier that hands the batch over.
// Every o and n · q is multiplied by q_scale.  Everything here is float32: gates, exponentials, sums, state.
//
// What a sequence keeps lies in one float32 row per (layer, slot), twice, `state` [slots][2][state_row]: per head the
// columns of S one after another, [V][K] (kind 2: [V + 1][K], the last column being n), and for kind 2 behind all heads
// the maximum m, [H][V + 1] (a copy per column, so that whoever owns a column reads nothing that another warp writes).
// A step reads the copy of the parity of the sequence's position at its start and writes the copy of the parity at its
// end, so a step of one token leaves what it read untouched and may run twice.
//
// The kernel: eight lanes share the rows of a column and a warp takes 4·NC columns, its part of the state in registers as
// pairs of rows (`fma.rn.f32x2`: two multiply-adds an instruction); a CTA of four warps takes 16·NC columns of a
// head of a sequence.  k, q, a and v of up to 32 tokens at a time arrive in shared memory by `cp.async` a batch ahead, and a
// token's rows are fetched from there while the token before is worked on.  The
// columns of a state never meet.  Sums over rows: kind 1 needs Sᵀk before it can go on (three exchanges among the eight
// lanes a token, with Sᵀq taken of the state before the write and u (k · q) added, so the read-out waits for nothing);
// the read-outs of eight tokens are summed together, seven exchanges for all eight, and lane r ends up with token r's.
// A step of single tokens has a kernel of its own (matrix_state_step) that reads and writes memory directly; both run the same
// arithmetic in the same order.
#include "common.cuh"
#include <type_traits>

namespace {
constexpr int MS_WARPS = 4;
constexpr int MS_MAX_BATCH = 32;       // a lane per token works out a batch's gates
constexpr int MS_DECAYED = 0, MS_DELTA = 1, MS_STABILIZED = 2, MS_FIXED = 3;
// kinds with a decay per head, key channel and token, kinds with two more numbers a token
constexpr bool ms_decays(int mode) { return mode == MS_DECAYED || mode == MS_DELTA; }
constexpr bool ms_numbers(int mode) { return mode == MS_DELTA || mode == MS_STABILIZED; }

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pk2(float lo, float hi) { f32x2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ float sum2(f32x2 v) { float lo, hi; asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); return lo + hi; }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) { f32x2 d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) { f32x2 d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) { f32x2 d; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }

__device__ __forceinline__ void ms_cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ms_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

struct MatrixStateArgs {
    const float *q, *k, *v, *decay, *s0, *s1;
    int ldq, ldk, ldv, ld_decay, ld_s0, ld_s1;
    float q_scale, cap;
    float* state;
    int state_row;
    const int *seq_slot, *seq_start, *seq_pos0;
    float* y;
    int ldy;
    float* den;
    int H, G, K, V, col_blocks, batch, vec_rows, vec_v, vec_state, max_new, warps, silu;
};

// log sigmoid(x), stable at both ends
__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

// A lane's part of the state: rows 4·(8j + r) … + 3 for j < NR/4 (as pairs) of NC columns from `my_col` on, from or into a copy
// of the state.  Rows and columns that do not exist are zero and stay so.
template <int NR, int NC>
__device__ __forceinline__ void load_state(f32x2 (&S)[NC][NR / 2], const float* base, int my_col, int VT, int K, int r, int vec) {
#pragma unroll
    for (int e = 0; e < NC; ++e) {
        const bool has = my_col + e < VT;
        const float* col = base + (size_t)(my_col + e) * K;
#pragma unroll
        for (int j = 0; j < NR / 4; ++j) {
            const int row = 4 * (8 * j + r);
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (has) {
                if (vec) { if (row < K) x = *reinterpret_cast<const float4*>(col + row); }
                else {
                    if (row < K) x.x = col[row];
                    if (row + 1 < K) x.y = col[row + 1];
                    if (row + 2 < K) x.z = col[row + 2];
                    if (row + 3 < K) x.w = col[row + 3];
                }
            }
            S[e][2 * j] = pk2(x.x, x.y);
            S[e][2 * j + 1] = pk2(x.z, x.w);
        }
    }
}
template <int NR, int NC>
__device__ __forceinline__ void store_state(const f32x2 (&S)[NC][NR / 2], float* base, int my_col, int VT, int K, int r, int vec) {
#pragma unroll
    for (int e = 0; e < NC; ++e) {
        if (my_col + e >= VT) continue;
        float* col = base + (size_t)(my_col + e) * K;
#pragma unroll
        for (int j = 0; j < NR / 4; ++j) {
            const int row = 4 * (8 * j + r);
            float x[4];
            asm("mov.b64 {%0, %1}, %2;" : "=f"(x[0]), "=f"(x[1]) : "l"(S[e][2 * j]));
            asm("mov.b64 {%0, %1}, %2;" : "=f"(x[2]), "=f"(x[3]) : "l"(S[e][2 * j + 1]));
            if (vec) { if (row < K) *reinterpret_cast<float4*>(col + row) = make_float4(x[0], x[1], x[2], x[3]); }
            else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (row + q < K) col[row + q] = x[q];
            }
        }
    }
}

// A token's rows as a lane holds them: k, q and (kinds 0 and 1) the decay at the lane's rows.
template <int NR> struct TokenRows { ulonglong2 k[NR / 4], q[NR / 4], d[NR / 4]; };

// One token: S moves on, and p gets the lane's share (its rows) of the read-outs.  a, b: kind 1 (b, k · q), kind 2 (what stays, what
// comes), kind 3 (what stays); v: the columns' values.
template <int MODE, int NR, int NC>
__device__ __forceinline__ void advance(f32x2 (&S)[NC][NR / 2], const TokenRows<NR>& X, const float (&v)[NC], float a, float b, int r, float (&p)[NC]) {
    constexpr int NV = NR / 4, NP = NR / 2;
    f32x2 dq[NC][2];
#pragma unroll
    for (int e = 0; e < NC; ++e) dq[e][0] = dq[e][1] = 0ull;
    if (MODE == MS_DELTA) {
        f32x2 dk[NC][2];
#pragma unroll
        for (int e = 0; e < NC; ++e) dk[e][0] = dk[e][1] = 0ull;
#pragma unroll
        for (int j = 0; j < NV; ++j)
#pragma unroll
            for (int e = 0; e < NC; ++e) {
                S[e][2 * j] = mul2(X.d[j].x, S[e][2 * j]);
                S[e][2 * j + 1] = mul2(X.d[j].y, S[e][2 * j + 1]);
                dk[e][0] = fma2(X.k[j].x, S[e][2 * j], dk[e][0]);
                dk[e][1] = fma2(X.k[j].y, S[e][2 * j + 1], dk[e][1]);
            }
        float d[NC];
#pragma unroll
        for (int e = 0; e < NC; ++e) d[e] = sum2(add2(dk[e][0], dk[e][1]));
#pragma unroll
        for (int o = 4; o > 0; o >>= 1)
#pragma unroll
            for (int e = 0; e < NC; ++e) d[e] += __shfl_xor_sync(0xffffffffu, d[e], o);
        // Sᵀq of the state before the write, while the exchanges are under way
#pragma unroll
        for (int j = 0; j < NV; ++j)
#pragma unroll
            for (int e = 0; e < NC; ++e) {
                dq[e][0] = fma2(X.q[j].x, S[e][2 * j], dq[e][0]);
                dq[e][1] = fma2(X.q[j].y, S[e][2 * j + 1], dq[e][1]);
            }
#pragma unroll
        for (int e = 0; e < NC; ++e) {
            const float u = a * (v[e] - d[e]);
            const f32x2 uu = pk2(u, u);
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                S[e][2 * j] = fma2(X.k[j].x, uu, S[e][2 * j]);
                S[e][2 * j + 1] = fma2(X.k[j].y, uu, S[e][2 * j + 1]);
            }
            p[e] = sum2(add2(dq[e][0], dq[e][1])) + (r == 0 ? u * b : 0.f);
        }
    } else {
        const f32x2 keep = pk2(a, a);
#pragma unroll
        for (int e = 0; e < NC; ++e) {
            const float w = MODE == MS_STABILIZED ? v[e] * b : v[e];
            const f32x2 ww = pk2(w, w);
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                S[e][2 * j] = fma2(X.k[j].x, ww, mul2(MODE == MS_DECAYED ? X.d[j].x : keep, S[e][2 * j]));
                S[e][2 * j + 1] = fma2(X.k[j].y, ww, mul2(MODE == MS_DECAYED ? X.d[j].y : keep, S[e][2 * j + 1]));
                dq[e][0] = fma2(X.q[j].x, S[e][2 * j], dq[e][0]);
                dq[e][1] = fma2(X.q[j].y, S[e][2 * j + 1], dq[e][1]);
            }
            p[e] = sum2(add2(dq[e][0], dq[e][1]));
        }
        (void)NP;
    }
}

// NR: rows of a column that a lane holds (K ≤ 8·NR; a multiple of 4); NC: columns a lane
template <int MODE, int NR, int NC>
__global__ void __launch_bounds__(MS_WARPS * 32, 1)
matrix_state_scan_kernel(const MatrixStateArgs A) {
    constexpr int KP = 8 * NR, NV = NR / 4;
    constexpr bool DECAY = ms_decays(MODE);
    constexpr int ROWS = DECAY ? 3 : 2;             // k, q (, decay)
    constexpr bool AHEAD = NR <= 16;                // a token's rows are fetched from shared memory while the one before is worked on
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ __align__(16) float ms_sm[];
    const int h = blockIdx.x / A.col_blocks, pb = blockIdx.x - h * A.col_blocks, s = blockIdx.y;
    const int slot = A.seq_slot[s];
    if (slot < 0) return;                           // padding (the whole CTA)
    const int start = A.seq_start[s], n = A.seq_start[s + 1] - start, pos0 = A.seq_pos0[s];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane & 7, c = lane >> 3, n_thr = blockDim.x;
    const int CW = (n_thr >> 5) * 4 * NC;           // columns of the CTA
    const int K = A.K, V = A.V, VT = V + (MODE == MS_STABILIZED ? 1 : 0), B = A.batch;
    const int g = h / (A.H / A.G);
    const int col0 = pb * CW + warp * 4 * NC;       // the warp's first column
    const bool active = col0 < VT;                  // (warps behind the last column only help to load)
    const int my_col = col0 + c * NC;
    const size_t copy_in = ((size_t)slot * 2 + (pos0 & 1)) * A.state_row, copy_out = ((size_t)slot * 2 + ((pos0 + n) & 1)) * A.state_row;
    const size_t head_at = (size_t)h * VT * K, max_at = (size_t)A.H * VT * K + (size_t)h * VT;

    // shared memory: per stage k, q (, decay) [B][KP] each and v [B][CW]; then per warp two numbers a token [B][2]
    const int stage_floats = B * (ROWS * KP + CW);
    float* scal = ms_sm + 2 * stage_floats + warp * B * 2;

    // rows K … KP − 1 stay zero in both stages
    if (K < KP) {
        for (int i = threadIdx.x; i < 2 * B * ROWS * (KP - K); i += n_thr) {
            const int row = i / (KP - K), cc = K + i - row * (KP - K);       // row: stage-major over [2][ROWS][B]
            const int st = row / (ROWS * B);
            ms_sm[st * stage_floats + (row - st * ROWS * B) * KP + cc] = 0.f;
        }
    }
    // who copies what: a thread's first token, column and step in tokens, for rows of K and of CW numbers in quads
    const bool whole_rows = A.vec_rows && n_thr % (K / 4) == 0;
    const int ii0 = whole_rows ? threadIdx.x / (K / 4) : 0, ii_step = whole_rows ? n_thr / (K / 4) : 1, q_col = (threadIdx.x - ii0 * (K / 4)) * 4;
    const int v0 = threadIdx.x / (CW / 4), v_step = n_thr / (CW / 4), v_col = (threadIdx.x - v0 * (CW / 4)) * 4;
    if (MODE == MS_STABILIZED && pb * CW <= V && V < pb * CW + CW) {        // the column of n takes k itself: its value is always 1
        for (int i = threadIdx.x; i < 2 * B; i += n_thr) ms_sm[(i / B) * stage_floats + ROWS * B * KP + (i % B) * CW + (V - pb * CW)] = 1.f;
    }
    auto fetch = [&](int i0, int st) {              // all threads: the inputs of the batch that begins at token i0
        const int nb = min(B, n - i0);
        float* ks = ms_sm + st * stage_floats;
        float* qs = ks + B * KP;
        float* ds = qs + B * KP;
        float* vs = ms_sm + st * stage_floats + ROWS * B * KP;
        const size_t t0 = (size_t)(start + i0);
        if (whole_rows) {                           // a thread's quads lie in one column of quads: no division here
            for (int ii = ii0; ii < nb; ii += ii_step) {
                ms_cp16(ks + ii * KP + q_col, A.k + (t0 + ii) * A.ldk + g * K + q_col);
                ms_cp16(qs + ii * KP + q_col, A.q + (t0 + ii) * A.ldq + g * K + q_col);
                if (DECAY) ms_cp16(ds + ii * KP + q_col, A.decay + (t0 + ii) * A.ld_decay + h * K + q_col);
            }
        } else if (A.vec_rows) {
            const int q4 = K / 4;
            for (int i = threadIdx.x; i < nb * q4; i += n_thr) {
                const int ii = i / q4, cc = (i - ii * q4) * 4;
                ms_cp16(ks + ii * KP + cc, A.k + (t0 + ii) * A.ldk + g * K + cc);
                ms_cp16(qs + ii * KP + cc, A.q + (t0 + ii) * A.ldq + g * K + cc);
                if (DECAY) ms_cp16(ds + ii * KP + cc, A.decay + (t0 + ii) * A.ld_decay + h * K + cc);
            }
        } else {
            for (int i = threadIdx.x; i < nb * K; i += n_thr) {
                const int ii = i / K, cc = i - ii * K;
                ms_cp4(ks + ii * KP + cc, A.k + (t0 + ii) * A.ldk + g * K + cc);
                ms_cp4(qs + ii * KP + cc, A.q + (t0 + ii) * A.ldq + g * K + cc);
                if (DECAY) ms_cp4(ds + ii * KP + cc, A.decay + (t0 + ii) * A.ld_decay + h * K + cc);
            }
        }
        if (A.vec_v) {                              // (V a multiple of 4: a group of four columns is whole or not there)
            if (pb * CW + v_col < V)
                for (int ii = v0; ii < nb; ii += v_step) ms_cp16(vs + ii * CW + v_col, A.v + (t0 + ii) * A.ldv + h * V + pb * CW + v_col);
        } else {
            for (int i = threadIdx.x; i < nb * CW; i += n_thr) {
                const int ii = i / CW, cc = i - ii * CW;
                if (pb * CW + cc < V) ms_cp4(vs + i, A.v + (t0 + ii) * A.ldv + h * V + pb * CW + cc);
            }
        }
    };
    // x · sigmoid(x) of this thread's own copies of a batch (the same places as in fetch)
    auto activate = [&](int nb, int st) {
        float* ks = ms_sm + st * stage_floats;
        float* qs = ks + B * KP;
        float* vs = ks + ROWS * B * KP;
        auto four = [](float* p) {
            float4 x = *reinterpret_cast<float4*>(p);
            x.x = silu_f(x.x); x.y = silu_f(x.y); x.z = silu_f(x.z); x.w = silu_f(x.w);
            *reinterpret_cast<float4*>(p) = x;
        };
        if (whole_rows) {
            for (int ii = ii0; ii < nb; ii += ii_step) { four(ks + ii * KP + q_col); four(qs + ii * KP + q_col); }
        } else if (A.vec_rows) {
            const int q4 = K / 4;
            for (int i = threadIdx.x; i < nb * q4; i += n_thr) {
                const int ii = i / q4, cc = (i - ii * q4) * 4;
                four(ks + ii * KP + cc);
                four(qs + ii * KP + cc);
            }
        } else {
            for (int i = threadIdx.x; i < nb * K; i += n_thr) {
                const int ii = i / K, at = ii * KP + i - ii * K;
                ks[at] = silu_f(ks[at]);
                qs[at] = silu_f(qs[at]);
            }
        }
        if (A.vec_v) {
            if (pb * CW + v_col < V)
                for (int ii = v0; ii < nb; ii += v_step) four(vs + ii * CW + v_col);
        } else {
            for (int i = threadIdx.x; i < nb * CW; i += n_thr)
                if (pb * CW + i % CW < V) vs[i] = silu_f(vs[i]);
        }
    };
    fetch(0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    f32x2 S[NC][NR / 2];
    load_state<NR, NC>(S, A.state + copy_in + head_at, my_col, VT, K, r, A.vec_state);
    // numbers of the batch's tokens: lane ii asks for token ii's, a batch ahead
    float m_run = 0.f, raw0 = 0.f, raw1 = 0.f;
    if (MODE == MS_STABILIZED && active) m_run = A.state[copy_in + max_at + col0];
    const float fixed = MODE == MS_FIXED ? A.decay[h] : 0.f;
    auto ask = [&](int i0) {
        const int ii = i0 + lane;
        raw0 = raw1 = 0.f;
        if (ms_numbers(MODE) && lane < B && ii < n) {
            raw0 = A.s0[(size_t)(start + ii) * A.ld_s0 + h];
            raw1 = A.s1[(size_t)(start + ii) * A.ld_s1 + (MODE == MS_DELTA ? g : h)];
        }
    };
    ask(0);
    for (int i0 = 0, st = 0; i0 < n; i0 += B, st ^= 1) {
        const int nb = min(B, n - i0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (MODE == MS_FIXED && A.silu) activate(nb, st);
        __syncthreads();                            // the batch lies in shared memory, and nobody reads the other stage any more
        if (i0 + B < n) fetch(i0 + B, st ^ 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        float floor_mine = 0.f;                     // kind 2: exp(−m) behind the lane's token
        if (MODE == MS_DELTA) {
            if (lane < B) { scal[2 * lane] = sigmoid_f(raw0); scal[2 * lane + 1] = raw1; }
        } else if (MODE == MS_STABILIZED) {
            const float log_i = A.cap * tanhf(raw0 / A.cap), log_f = log_sigmoid(A.cap * tanhf(raw1 / A.cap));
            // m of every token by a scan over the lanes: from m before lane's token and the ones ahead of it, m becomes
            // max(sum_f + m, top), and two such steps one after the other are a step of the same form
            float sum_f = lane < nb ? log_f : 0.f, top = lane < nb ? log_i : -INFINITY;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float pf = __shfl_up_sync(0xffffffffu, sum_f, o), pt = __shfl_up_sync(0xffffffffu, top, o);
                if (lane >= o) { top = fmaxf(pt + sum_f, top); sum_f += pf; }
            }
            const float behind = fmaxf(sum_f + m_run, top);
            float before = __shfl_up_sync(0xffffffffu, behind, 1);
            if (lane == 0) before = m_run;
            m_run = __shfl_sync(0xffffffffu, behind, 31);
            if (lane < B) { scal[2 * lane] = expf(log_f + before - behind); scal[2 * lane + 1] = expf(log_i - behind); }
            floor_mine = expf(-behind);
        }
        ask(i0 + B);
        __syncwarp();
        if (!active) continue;                      // (whole warps)
        const float* ks = ms_sm + st * stage_floats + 4 * r;
        const float* vs = ms_sm + st * stage_floats + ROWS * B * KP + warp * 4 * NC + c * NC;
        auto rows_of = [&](int ii, TokenRows<NR>& X) {
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                X.k[j] = *reinterpret_cast<const ulonglong2*>(ks + ii * KP + 32 * j);
                if (DECAY) X.d[j] = *reinterpret_cast<const ulonglong2*>(ks + (2 * B + ii) * KP + 32 * j);
                X.q[j] = *reinterpret_cast<const ulonglong2*>(ks + (B + ii) * KP + 32 * j);
            }
        };
        TokenRows<NR> X[AHEAD ? 2 : 1];
        if (AHEAD) rows_of(0, X[0]);
        // eight tokens from e0 on; FULL: all eight are there (nothing then stands between one token's loads and the next's)
        auto eight = [&](int e0, auto full) {
            constexpr bool FULL = decltype(full)::value;
            float p[8][NC];                         // this lane's share of the read-outs of eight tokens
#pragma unroll
            for (int t = 0; t < 8; ++t) {
                const int ii = e0 + t;
                if (FULL || ii < nb) {              // (uniform over the CTA)
                    if (AHEAD) rows_of((FULL && t < 7) || ii + 1 < nb ? ii + 1 : ii, X[(t + 1) & 1]);
                    else rows_of(ii, X[0]);
                    float v[NC];
#pragma unroll
                    for (int e = 0; e < NC; ++e) v[e] = vs[ii * CW + e];     // (columns that do not exist: anything, it goes nowhere)
                    float2 ab = make_float2(fixed, 0.f);
                    if (ms_numbers(MODE)) ab = *reinterpret_cast<const float2*>(scal + 2 * ii);
                    advance<MODE, NR, NC>(S, X[AHEAD ? (t & 1) : 0], v, ab.x, ab.y, r, p[t]);
                } else {
#pragma unroll
                    for (int e = 0; e < NC; ++e) p[t][e] = 0.f;
                }
            }
            // eight sums over eight lanes: each exchange halves the tokens a lane is responsible for
            float o[NC];
#pragma unroll
            for (int e = 0; e < NC; ++e) {
#pragma unroll
                for (int w = 4; w > 0; w >>= 1) {
                    const bool up = r & w;
#pragma unroll
                    for (int t = 0; t < w; ++t) {
                        const float give = up ? p[t][e] : p[t + w][e], mine = up ? p[t + w][e] : p[t][e];
                        p[t][e] = mine + __shfl_xor_sync(0xffffffffu, give, w);
                    }
                }
                o[e] = p[0][e] * A.q_scale;
            }
            const int ii = e0 + r;
            const float em = MODE == MS_STABILIZED ? __shfl_sync(0xffffffffu, floor_mine, ii & 31) : 0.f;
            if (FULL || ii < nb) {
                const size_t row = (size_t)(start + i0 + ii);
#pragma unroll
                for (int e = 0; e < NC; ++e) {
                    if (my_col + e < V) A.y[row * A.ldy + (size_t)h * V + my_col + e] = o[e];
                    else if (MODE == MS_STABILIZED && my_col + e == V) {
                        A.den[(row * A.H + h) * 2] = o[e];
                        A.den[(row * A.H + h) * 2 + 1] = em;
                    }
                }
            }
        };
        for (int e0 = 0; e0 < nb; e0 += 8) {
            if (nb - e0 >= 8) eight(e0, std::true_type{});
            else eight(e0, std::false_type{});
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (!active) return;
    store_state<NR, NC>(S, A.state + copy_out + head_at, my_col, VT, K, r, A.vec_state);
    if (MODE == MS_STABILIZED && r == 0) {
#pragma unroll
        for (int e = 0; e < NC; ++e)
            if (my_col + e < VT) A.state[copy_out + max_at + my_col + e] = m_run;
    }
}

// A step of single tokens: a warp takes 4·NC columns of a head of a sequence, straight from and into device memory (no other
// warp shares enough of a token's rows to be worth a stage in shared memory).  The same arithmetic in the same order.
template <int MODE, int NR, int NC>
__global__ void __launch_bounds__(MS_WARPS * 32)
matrix_state_step_kernel(const MatrixStateArgs A) {
    constexpr int NV = NR / 4;
    constexpr bool DECAY = ms_decays(MODE);
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.y, slot = A.seq_slot[s];
    if (slot < 0) return;                           // padding
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane & 7, c = lane >> 3;
    const int unit = blockIdx.x * MS_WARPS + warp;
    const int h = unit / A.col_blocks;
    if (h >= A.H) return;                           // (whole warps; no block-wide barrier below)
    const int K = A.K, V = A.V, VT = V + (MODE == MS_STABILIZED ? 1 : 0), g = h / (A.H / A.G);
    const int col0 = (unit - h * A.col_blocks) * 4 * NC, my_col = col0 + c * NC;
    const int pos0 = A.seq_pos0[s];
    const size_t t = (size_t)A.seq_start[s];
    const size_t copy_in = ((size_t)slot * 2 + (pos0 & 1)) * A.state_row, copy_out = ((size_t)slot * 2 + ((pos0 + 1) & 1)) * A.state_row;
    const size_t head_at = (size_t)h * VT * K, max_at = (size_t)A.H * VT * K + (size_t)h * VT;
    f32x2 S[NC][NR / 2];
    load_state<NR, NC>(S, A.state + copy_in + head_at, my_col, VT, K, r, A.vec_state);
    TokenRows<NR> X;
    auto row_of = [&](const float* base, ulonglong2 (&out)[NV]) {
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int row = 4 * (8 * j + r);
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (A.vec_rows) { if (row < K) x = *reinterpret_cast<const float4*>(base + row); }
            else {
                if (row < K) x.x = base[row];
                if (row + 1 < K) x.y = base[row + 1];
                if (row + 2 < K) x.z = base[row + 2];
                if (row + 3 < K) x.w = base[row + 3];
            }
            out[j].x = pk2(x.x, x.y);
            out[j].y = pk2(x.z, x.w);
        }
    };
    row_of(A.k + t * A.ldk + (size_t)g * K, X.k);
    row_of(A.q + t * A.ldq + (size_t)g * K, X.q);
    if (DECAY) row_of(A.decay + t * A.ld_decay + (size_t)h * K, X.d);
    const bool act = MODE == MS_FIXED && A.silu;
    if (act) {
        auto both = [](unsigned long long& x) {
            float lo, hi;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(x));
            x = pk2(silu_f(lo), silu_f(hi));
        };
#pragma unroll
        for (int j = 0; j < NV; ++j) { both(X.k[j].x); both(X.k[j].y); both(X.q[j].x); both(X.q[j].y); }
    }
    float v[NC], p[NC];
#pragma unroll
    for (int e = 0; e < NC; ++e)
        v[e] = my_col + e < V ? A.v[t * A.ldv + (size_t)h * V + my_col + e] : (MODE == MS_STABILIZED && my_col + e == V) ? 1.f : 0.f;
    if (act) {
#pragma unroll
        for (int e = 0; e < NC; ++e) v[e] = silu_f(v[e]);
    }
    float a = MODE == MS_FIXED ? A.decay[h] : 0.f, b = 0.f, m_new = 0.f;
    if (MODE == MS_DELTA) {
        a = sigmoid_f(A.s0[t * A.ld_s0 + h]);
        b = A.s1[t * A.ld_s1 + g];
    } else if (MODE == MS_STABILIZED) {
        const float m_run = A.state[copy_in + max_at + col0];
        const float log_i = A.cap * tanhf(A.s0[t * A.ld_s0 + h] / A.cap), log_f = log_sigmoid(A.cap * tanhf(A.s1[t * A.ld_s1 + h] / A.cap));
        m_new = fmaxf(log_f + m_run, log_i);
        a = expf(log_f + m_run - m_new);
        b = expf(log_i - m_new);
    }
    advance<MODE, NR, NC>(S, X, v, a, b, r, p);
    store_state<NR, NC>(S, A.state + copy_out + head_at, my_col, VT, K, r, A.vec_state);
#pragma unroll
    for (int e = 0; e < NC; ++e) {
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) p[e] += __shfl_xor_sync(0xffffffffu, p[e], o);
        if (r != 0) continue;
        if (my_col + e < V) A.y[t * A.ldy + (size_t)h * V + my_col + e] = p[e] * A.q_scale;
        else if (MODE == MS_STABILIZED && my_col + e == V) {
            A.den[(t * A.H + h) * 2] = p[e] * A.q_scale;
            A.den[(t * A.H + h) * 2 + 1] = expf(-m_new);
        }
        if (MODE == MS_STABILIZED && my_col + e < VT) A.state[copy_out + max_at + my_col + e] = m_new;
    }
}

template <int MODE, int NR, int NC> int launch_scan(MatrixStateArgs& A, int n_seqs, cudaStream_t stream) {
    constexpr int KP = 8 * NR, ROWS = ms_decays(MODE) ? 3 : 2;
    const int VT = A.V + (MODE == MS_STABILIZED ? 1 : 0), chunks = (VT + 4 * NC - 1) / (4 * NC);
    if (A.max_new == 1) {
        A.col_blocks = chunks;
        launch_chained(matrix_state_step_kernel<MODE, NR, NC>, dim3((A.H * chunks + MS_WARPS - 1) / MS_WARPS, n_seqs), dim3(MS_WARPS * 32), (size_t)0,
                       stream, A);
        return vlrf_check_launch("matrix_state_step");
    }
    const int warps = A.warps, CW = warps * 4 * NC;
    A.col_blocks = (chunks + warps - 1) / warps;
    // tokens a batch: as many as the step's longest run has, at most 16, fewer where the rows are long
    const auto bytes = [&](int b) { return (size_t)(2 * b * (ROWS * KP + CW) + warps * b * 2) * sizeof(float); };
    while (A.batch > 1 && bytes(A.batch) > 110 * 1024) A.batch /= 2;
    const size_t smem = bytes(A.batch);
    static size_t allowed = 48 * 1024;
    if (smem > allowed) {
        const cudaError_t e = cudaFuncSetAttribute(matrix_state_scan_kernel<MODE, NR, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return vlrf_fail(VLRF_ERR_CUDA, "matrix_state_scan: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        allowed = smem;
    }
    launch_chained(matrix_state_scan_kernel<MODE, NR, NC>, dim3(A.H * A.col_blocks, n_seqs), dim3(warps * 32), smem, stream, A);
    return vlrf_check_launch("matrix_state_scan");
}

template <int MODE> int pick_scan(MatrixStateArgs& A, int nc, int n_seqs, cudaStream_t stream) {
#define GO(NR) return nc == 1 ? launch_scan<MODE, NR, 1>(A, n_seqs, stream) : nc == 2 ? launch_scan<MODE, NR, 2>(A, n_seqs, stream) : launch_scan<MODE, NR, 4>(A, n_seqs, stream)
    if (A.K <= 32) GO(4);
    if (A.K <= 64) GO(8);
    if (A.K <= 128) GO(16);
#undef GO
    if (A.K <= 256) return nc == 1 ? launch_scan<MODE, 32, 1>(A, n_seqs, stream) : launch_scan<MODE, 32, 2>(A, n_seqs, stream);
    return launch_scan<MODE, 64, 1>(A, n_seqs, stream);
}

bool on16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
int ms_forced_columns = 0, ms_forced_warps = 0;
}  // namespace

// For measurements and tests: a lane's columns (1, 2 or 4) and a CTA's warps (1, 2 or 4); 0: chosen by the step's size.
extern "C" int vlrf_matrix_state_force(int columns, int warps) {
    VLRF_REQUIRE(columns == 0 || columns == 1 || columns == 2 || columns == 4, "matrix_state_scan: a lane takes 1, 2 or 4 columns, not %d", columns);
    VLRF_REQUIRE(warps == 0 || warps == 1 || warps == 2 || warps == 4, "matrix_state_scan: a CTA has 1, 2 or 4 warps, not %d", warps);
    ms_forced_columns = columns;
    ms_forced_warps = warps;
    return VLRF_OK;
}

extern "C" int vlrf_matrix_state_scan(int kind, const float* q, int ldq, const float* k, int ldk, const float* v, int ldv,
                                      const float* decay, int ld_decay, const float* s0, int ld_s0, const float* s1, int ld_s1,
                                      float q_scale, float cap, float* state, int state_row, const int* seq_slot,
                                      const int* seq_start, const int* seq_pos0, float* y, int ldy, float* den, int n_seqs, int max_new,
                                      int H, int G, int K, int V, int input_act, cudaStream_t stream) {
    VLRF_REQUIRE(kind >= MS_DECAYED && kind <= MS_FIXED, "matrix_state_scan: unknown kind %d", kind);
    VLRF_REQUIRE(n_seqs >= 0 && max_new >= 0 && H > 0 && G > 0 && K > 0 && V > 0 && H % G == 0, "matrix_state_scan: bad sizes (heads %d/%d, state %d by %d)", H, G, K, V);
    VLRF_REQUIRE(K <= 512 && V <= 4096 && n_seqs <= 65535, "matrix_state_scan: a state of %d rows by %d columns is above 512 by 4096, or too many sequences", K, V);
    VLRF_REQUIRE(ldq >= G * K && ldk >= G * K && ldv >= H * V && ldy >= H * V, "matrix_state_scan: columns lie outside the rows");
    VLRF_REQUIRE(input_act == VLRF_ACT_NONE || (input_act == VLRF_ACT_SILU && kind == MS_FIXED), "matrix_state_scan: input activation %d is not taken by kind %d", input_act, kind);
    VLRF_REQUIRE(kind != MS_FIXED || decay != nullptr, "matrix_state_scan: this kind needs a decay per head");
    VLRF_REQUIRE(!ms_decays(kind) || (decay != nullptr && ld_decay >= H * K), "matrix_state_scan: this kind needs a decay per head and key channel");
    VLRF_REQUIRE(!ms_numbers(kind) || (s0 != nullptr && s1 != nullptr && ld_s0 >= H && ld_s1 >= (kind == MS_DELTA ? G : H)), "matrix_state_scan: this kind needs two numbers a token");
    VLRF_REQUIRE(kind != MS_STABILIZED || (den != nullptr && cap > 0.f), "matrix_state_scan: this kind needs a place for the denominators and a positive cap");
    const long long need = kind == MS_STABILIZED ? (long long)H * (V + 1) * (K + 1) : (long long)H * V * K;
    VLRF_REQUIRE(need <= state_row, "matrix_state_scan: the state row of %d numbers is shorter than %lld", state_row, need);
    if (n_seqs == 0 || max_new == 0) return VLRF_OK;
    MatrixStateArgs A;
    A.q = q; A.k = k; A.v = v; A.decay = decay; A.s0 = s0; A.s1 = s1;
    A.ldq = ldq; A.ldk = ldk; A.ldv = ldv; A.ld_decay = ld_decay; A.ld_s0 = ld_s0; A.ld_s1 = ld_s1;
    A.q_scale = q_scale; A.cap = cap; A.state = state; A.state_row = state_row;
    A.seq_slot = seq_slot; A.seq_start = seq_start; A.seq_pos0 = seq_pos0;
    A.y = y; A.ldy = ldy; A.den = den; A.H = H; A.G = G; A.K = K; A.V = V; A.col_blocks = 1;
    A.max_new = max_new; A.silu = input_act == VLRF_ACT_SILU; A.warps = ms_forced_warps ? ms_forced_warps : 4;
    A.batch = max_new < MS_MAX_BATCH ? max_new : MS_MAX_BATCH;
    A.vec_rows = K % 4 == 0 && on16(q) && on16(k) && ldq % 4 == 0 && ldk % 4 == 0 && (!ms_decays(kind) || (on16(decay) && ld_decay % 4 == 0));
    A.vec_v = V % 4 == 0 && on16(v) && ldv % 4 == 0;
    A.vec_state = K % 4 == 0 && on16(state) && state_row % 4 == 0;
    // columns a lane (measured): single tokens 2; prompts 1 where the step's columns are fewer than warps for every scheduler of
    // the GPU, else 2; 4 for the decayed kind with columns in plenty (it has the most rows to read from shared memory)
    int sms = 148, dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    const long long warps1 = (long long)n_seqs * H * ((V + 3) / 4);
    int nc = ms_forced_columns ? ms_forced_columns : max_new == 1 ? 2 : warps1 <= 4LL * sms ? 1 : (kind == MS_DECAYED && warps1 > 8LL * sms) ? 4 : 2;
    if (K > 128 && nc > 2) nc = 2;
    switch (kind) {
        case MS_DECAYED: return pick_scan<MS_DECAYED>(A, nc, n_seqs, stream);
        case MS_DELTA: return pick_scan<MS_DELTA>(A, nc, n_seqs, stream);
        case MS_FIXED: return pick_scan<MS_FIXED>(A, nc, n_seqs, stream);
        default: return pick_scan<MS_STABILIZED>(A, nc, n_seqs, stream);
    }
}
