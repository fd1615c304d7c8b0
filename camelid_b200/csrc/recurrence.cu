// Recurrent mixers with a matrix state per head: S [key_dim, value_dim] in float, carried from
// token to token for each sequence.
//
//   gated delta rule (one decay per key channel, or one per head):  S <- diag(g) S;  u = beta (v - S^T k);
//                                                  S <- S + k u^T;  o = S^T q
//   matrix memory with exponential gates:          m' = max(f + m, i);
//                                                  S <- e^(f + m - m') S + e^(i - m') k v^T  (n likewise with k alone);
//                                                  o = S^T q / (max(|n . q|, e^(-m')) + 1e-6)
//
//   retention (a fixed decay per head):            S <- d S + k v^T;  o = S^T q
//   state-space recurrence (decay e^(-e^A dt) and step dt per head and token, k and q shared by groups of heads):
//                                                  S <- e^(-e^A dt) S + dt k v^T;  o = S^T q + D v
//   generalized delta rule (decay w and removal rate a per key channel, u = k / |k|):
//                                                  S <- diag(w) S - (a * u)(u^T S) + k v^T;  o = S^T r
//
// All are independent per column of S: eight threads of a warp share one column (a slice of
// the key axis each, in registers) of one (sequence, head) and walk the sequence's new tokens
// in order, so a prompt's rows and the same rows fed one by one are summed in the same order.
// The matrix memory keeps n as one more column (whose v is 1) and a copy of m per column, so
// that no thread reads what another writes. q, k, gates of a few tokens at a time are staged
// in shared memory by the whole block.
//
// Before them: the short causal convolution with SiLU and the unit norm of q and k for the
// delta rule. After them: the per-head RMS norm with weight and sigmoid gate.
#include "common.cuh"

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float logsigmoid_f(float x) { return x < 0.f ? x - log1pf(expf(x)) : -log1pf(expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float split_sum(const float* p, int n, long stride) {
    float v = p[0];
    for (int s0 = 1; s0 < n; s0 += 8) {                        // eight splits' loads in flight, added in split order
        float t[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) t[k] = p[(size_t)min(s0 + k, n - 1) * stride];
#pragma unroll
        for (int k = 0; k < 8; ++k) v += s0 + k < n ? t[k] : 0.f;
    }
    return v;
}

// ------------------------------------------------------------------------------------
// Short convolution + SiLU (+ unit norm). `proj` [rows, ld] holds, from column 0, the q
// channels (qk_heads x key_dim), the k channels (the same) and the v channels (heads x
// value_dim) before the convolution; `conv_w` [channels, taps] float, the last tap the current
// token's; `state` [slots, taps - 1, channels] the inputs of the tokens before the step.
// A warp owns one (row, head of q | k | v). q and k become x / sqrt(sum x^2 + 1e-6), q times
// q_scale. out [rows, channels] float. With `update_state` (steps in which every sequence brings
// one row) the warp also moves its channels of the state on by that row; otherwise a later
// launch replaces the state.
__global__ void conv_unit_kernel(const float* __restrict__ proj, long ld, const float* __restrict__ conv_w,
                                 float* __restrict__ state, int update_state, const int* __restrict__ row_seq,
                                 const int* __restrict__ row_pos, const int* __restrict__ seq_row0,
                                 const int* __restrict__ seq_slot, float* __restrict__ out, int rows, int qk_heads,
                                 int heads, int key_dim, int value_dim, int taps, float q_scale,
                                 const float* __restrict__ decay_in, long ldd, const float* __restrict__ a_log,
                                 const float* __restrict__ dt_bias, float* __restrict__ decay_out, int decay_dim) {
    pdl_wait();
    pdl_launch_dependents();
    const int units = 2 * qk_heads + heads + (decay_in ? heads : 0);
    const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    if (warp >= rows * units) return;
    const int r = warp / units, u = warp % units;
    if (u >= 2 * qk_heads + heads) {
        // the decays of one (row, head), once for all the scan's blocks of that head:
        // g = exp(-exp(a_log[head]) softplus(x + dt_bias))
        const int hd = u - 2 * qk_heads - heads;
        const float rate = expf(a_log[hd]);
        for (int d = lane; d < decay_dim; d += 32) {            // decay_dim: key_dim (a decay per channel) or 1 (per head)
            const float x = decay_in[(size_t)r * ldd + hd * decay_dim + d] + dt_bias[hd * decay_dim + d];
            decay_out[((size_t)r * heads + hd) * decay_dim + d] = expf(-rate * softplus_f(x));
        }
        return;
    }
    const int channels = 2 * qk_heads * key_dim + heads * value_dim;
    int c0, n;
    if (u < 2 * qk_heads) { c0 = u * key_dim; n = key_dim; }
    else { c0 = 2 * qk_heads * key_dim + (u - 2 * qk_heads) * value_dim; n = value_dim; }
    const int s = row_seq[r], pos = row_pos[r], inside = r - seq_row0[s];
    float* st = state + (size_t)seq_slot[s] * (taps - 1) * channels;
    float ss = 0.f;
    // A lane's channels eight at a time, tap by tap: the eight loads of a tap are unconditional (of a valid
    // place) and in flight together; nothing is stored until every tap has been read.
    for (int base = c0; base < c0 + n; base += 256) {
        float acc[8];
        int cc[8];
        bool ok[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const int c = base + lane + 32 * e;
            ok[e] = c < c0 + n;
            cc[e] = ok[e] ? c : c0;
            acc[e] = 0.f;
        }
        const int ne = min(8, (c0 + n - base + 31) / 32);  // groups of 32 channels that are there at all (the same for the warp)
        for (int j = 0; j < taps; ++j) {
            const int back = taps - 1 - j;                 // tokens before this one
            if (back > pos) continue;                      // before the sequence's start
            const float* src = back <= inside ? proj + (size_t)(r - back) * ld : st + (size_t)(taps - 1 + inside - back) * channels;
            float x[8], w[8];
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (e < ne) { x[e] = src[cc[e]]; w[e] = conv_w[(size_t)cc[e] * taps + j]; }
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (e < ne) acc[e] = fmaf(w[e], x[e], acc[e]);
        }
        if (update_state && taps > 1) {                    // one row per sequence: drop the oldest input, keep this one
            for (int j = 0; j + 2 < taps; ++j) {
                float t[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) t[e] = st[(size_t)(j + 1) * channels + cc[e]];
#pragma unroll
                for (int e = 0; e < 8; ++e)
                    if (ok[e]) st[(size_t)j * channels + cc[e]] = pos + j + 2 >= taps ? t[e] : 0.f;
            }
            float t[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) t[e] = proj[(size_t)r * ld + cc[e]];
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (ok[e]) st[(size_t)(taps - 2) * channels + cc[e]] = t[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            if (!ok[e]) continue;
            const float a = silu_f(acc[e]);
            out[(size_t)r * channels + cc[e]] = a;
            ss = fmaf(a, a, ss);
        }
    }
    if (u < 2 * qk_heads) {
        ss = warp_sum(ss);
        const float scale = (u < qk_heads ? q_scale : 1.0f) / sqrtf(ss + 1e-6f);
        __syncwarp();
        for (int c = c0 + lane; c < c0 + n; c += 32) out[(size_t)r * channels + c] *= scale;
    }
}

// decay_in (may be null) [rows, ldd] (heads x decay_dim, decay_dim = key_dim or 1): the decays' inputs; decay_out [rows, heads x decay_dim] gets
// g = exp(-exp(a_log[head]) softplus(x + dt_bias)), what the delta-rule scan multiplies its state by.
extern "C" int cml_conv_unit(const float* proj, long ld, const float* conv_w, float* state, int update_state, const int* row_seq,
                             const int* row_pos, const int* seq_row0, const int* seq_slot, float* out, int rows, int qk_heads,
                             int heads, int key_dim, int value_dim, int taps, float q_scale, const float* decay_in, long ldd,
                             const float* a_log, const float* dt_bias, float* decay_out, int decay_dim, void* stream) {
    if (rows <= 0) return 0;
    if (taps < 1 || (decay_in && decay_dim != 1 && decay_dim != key_dim)) return CML_ERR_BAD_SIZE;
    const long warps = (long)rows * (2 * qk_heads + heads + (decay_in ? heads : 0));
    launch_pdl(conv_unit_kernel, dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, (cudaStream_t)stream, proj, ld, conv_w, state,
               update_state, row_seq, row_pos, seq_row0, seq_slot, out, rows, qk_heads, heads, key_dim, value_dim, taps, q_scale, decay_in, ldd,
               a_log, dt_bias, decay_out, decay_dim);
    return cml_launch_status();
}

// ------------------------------------------------------------------------------------
// The scans. A block of 128 threads owns 128 / NS columns of one (sequence, head); the key axis of a
// column is cut into NS slices (a power of two up to 32) of DS channels, one thread each, the NS
// threads of a column in one warp (lane = NS * column + slice), so that a dot product over the key
// axis is DS multiply-adds and a butterfly of log2 NS shuffles, always in the same order, whatever
// the step or the batch. The delta rule takes its two products
// (with k for the write, with q for the read-out) from the decayed state at once and adds the
// write's share u (k . q) to the read-out, so a token waits only for the write of the one before. The state lies column by column
// ([.., column, key channel]): a warp reads and writes whole rows of it with 16-byte accesses.
// q, k and the decays of SCAN_TOKENS tokens at a time stand in shared memory (slices padded by
// four floats against bank conflicts); the next tokens' values are fetched into registers
// while these are worked on.
//
// MODE 0, gated delta rule. in_a = qkv [rows, lda]: unit q (qk_heads x D), unit k, v (heads x Dv)
// from conv_unit_kernel; in_b [rows, ldb]: beta before the sigmoid at column b_col + head;
// in_c [rows, ldc] (heads x D, or heads with one decay per head): the decays g (decay_ready), or their input:
// g = exp(-exp(a_log[head]) softplus(x + dt_bias)).
// state [slots, heads, Dv, D]. out [rows, heads x Dv] = S^T q.
// MODE 1, matrix memory. in_a = proj [rows, lda] with q at q_col (heads x D), k at k_col, v at
// v_col (heads x Dv), gate inputs at i_col + head and f_col + head (before bias and cap).
// state [slots, heads, Dv + 1, D] (column Dv is n), state_m [slots, heads, Dv + 1] (m, one copy
// per column, so that no thread reads what another writes). out [rows, heads, Dv + 2]: S^T q per
// column, then n . q, then m after the token.
// MODE 2, retention. in_a = proj [rows, lda] with q at q_col (heads x D), k at k_col, v at v_col (heads x Dv), q and k
// turned and scaled already; vec_a [heads]: the heads' decays. state [slots, heads, Dv, D]. out [rows, heads x Dv].
// MODE 3, state-space recurrence. in_a [rows, lda] from ssm_inputs_kernel: v at v_col (heads x Dv), k and q at k_col and q_col
// (qk_heads x D, each shared by heads / qk_heads heads); in_b [rows, ldb]: the steps dt (heads), then the decays
// (heads); vec_a [heads]: D. state [slots, heads, Dv, D]. out [rows, heads x Dv].
#define SCAN_TOKENS 8

struct ScanParams {
    const float* in_a; long lda;
    const float* in_b; long ldb; int b_col;
    const float* in_c; long ldc;
    const float* vec_a;           // a_log [heads]            | input-gate bias [heads]
    const float* vec_b;           // dt_bias [heads x D]      | forget-gate bias [heads]
    float* state; float* state_m;
    const int* seq_row0; const int* seq_new; const int* seq_start; const int* seq_slot;
    float* out;
    int heads, qk_heads, D, Dv;
    int q_col, k_col, v_col, i_col, f_col;
    float cap, q_scale;
    int decay_ready;              // in_c holds the decays themselves (conv_unit_kernel made them)
    int decay_dim;                // D: one decay per key channel; 1: one per head (in_c and vec_b are heads x decay_dim)
};

template <int NS>
__device__ __forceinline__ float slices_sum(float v) {
#pragma unroll
    for (int sh = 1; sh < NS; sh <<= 1) v += __shfl_xor_sync(0xffffffffu, v, sh);
    return v;
}

template <int DS, int MODE, int NS>
__global__ void __launch_bounds__(128) scan_kernel(const ScanParams p) {
    constexpr int SCAN_COLS = 128 / NS;                // columns of a block
    constexpr int DPAD = NS * DS;                      // key channels a block can take
    constexpr int SL = DS == 4 ? 4 : DS + 4;           // floats of a slice in shared memory (padded against bank conflicts)
    constexpr int PER = SCAN_TOKENS * DPAD / 128;      // staged values per thread and array
    __shared__ __align__(16) float sq[SCAN_TOKENS][NS * SL], sk[SCAN_TOKENS][NS * SL], sg[MODE == 0 ? SCAN_TOKENS : 1][NS * SL];
    __shared__ float sv[SCAN_TOKENS][SCAN_COLS], s1[SCAN_TOKENS], s2[SCAN_TOKENS], skq[SCAN_TOKENS];
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, hd = blockIdx.y;
    const int D = p.D, Dv = p.Dv, heads = p.heads;
    const int cols = MODE == 1 ? Dv + 1 : Dv;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int slice = lane % NS;
    const int wcol = warp * (32 / NS) + lane / NS;       // this thread's column within the block
    const int c = blockIdx.z * SCAN_COLS + wcol;
    const bool live = c < cols;
    const int d0 = slice * DS;
    const int row0 = p.seq_row0[s], n = p.seq_new[s];
    const bool fresh = p.seq_start[s] == 0;
    const size_t cell = ((size_t)p.seq_slot[s] * heads + hd) * cols + (live ? c : 0);
    float* st = p.state + cell * D;
    const bool vec = (D & 3) == 0;
    float S[DS];
#pragma unroll
    for (int i = 0; i < DS; i += 4) {
        if (live && !fresh && vec && d0 + i < D) {
            const float4 t = *reinterpret_cast<const float4*>(st + d0 + i);
            S[i] = t.x; S[i + 1] = t.y; S[i + 2] = t.z; S[i + 3] = t.w;
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) S[i + j] = (live && !fresh && d0 + i + j < D) ? st[d0 + i + j] : 0.f;
        }
    }
    float m = 0.f;
    if (MODE == 1 && live && !fresh) m = p.state_m[cell];
    const float keep = MODE >= 2 ? p.vec_a[hd] : 0.f;          // retention: the head's decay; state space: its D
    const int g = (MODE == 0 || MODE == 3) ? hd / (heads / p.qk_heads) : hd;
    const int qc = MODE == 0 ? g * D : p.q_col + g * D;
    const int kc = MODE == 0 ? (p.qk_heads + g) * D : p.k_col + g * D;
    const int vc = MODE == 0 ? 2 * p.qk_heads * D + hd * Dv : p.v_col + hd * Dv;
    const float a_rate = (MODE == 0 && !p.decay_ready) ? expf(p.vec_a[hd]) : 0.f;
    const bool head_decay = MODE == 0 && p.decay_dim == 1;      // one decay per head: a number per token (s2), not a row of sg
    // staging: thread -> (token, key channel) of each array, one value of v, and the scalars
    // Nothing uses a fetched value before `stage`: a use right behind its load would hold the warp until the
    // load is back, once per round, instead of behind the tokens in between.
    float rq[PER], rk[PER], rg[MODE == 0 ? PER : 1], rv = 0.f, r1 = 0.f, r2 = 0.f;
    float bias[MODE == 0 ? PER : 1];                   // dt_bias of the channels this thread stages (the same every round)
    if (MODE == 0 && !p.decay_ready) {
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            const int d = (threadIdx.x + 128 * e) % DPAD;
            bias[e] = p.vec_b[head_decay ? hd : hd * D + (d < D ? d : 0)];
        }
    }
    auto fetch = [&](int t0) {
        const int nt = min(SCAN_TOKENS, n - t0);
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            const int idx = threadIdx.x + 128 * e, t = idx / DPAD, d = idx % DPAD;
            const bool ok = t < nt && d < D;
            const size_t r = (size_t)(row0 + t0 + (ok ? t : 0));
            const int dd = ok ? d : 0;
            rq[e] = p.in_a[r * p.lda + qc + dd];
            rk[e] = p.in_a[r * p.lda + kc + dd];
            if (MODE == 0 && !head_decay) rg[e] = p.in_c[r * p.ldc + hd * D + dd];
        }
        if (threadIdx.x < SCAN_TOKENS * SCAN_COLS) {
            const int t = threadIdx.x / SCAN_COLS, cc = blockIdx.z * SCAN_COLS + threadIdx.x % SCAN_COLS;
            const bool ok = t < nt && cc < Dv;
            rv = p.in_a[(size_t)(row0 + t0 + (ok ? t : 0)) * p.lda + vc + (ok ? cc : 0)];
        }
        if (threadIdx.x < SCAN_TOKENS) {
            const size_t r = (size_t)(row0 + t0 + (threadIdx.x < nt ? threadIdx.x : 0));
            if (MODE == 0) {
                r1 = p.in_b[r * p.ldb + p.b_col + hd];
                if (head_decay) r2 = p.in_c[r * p.ldc + hd];
            } else if (MODE == 1) { r1 = p.in_a[r * p.lda + p.i_col + hd]; r2 = p.in_a[r * p.lda + p.f_col + hd]; }
            else if (MODE == 3) { r1 = p.in_b[r * p.ldb + hd]; r2 = p.in_b[r * p.ldb + heads + hd]; }
        }
        // The loads stay here, ahead of the tokens that are worked on meanwhile: without this the compiler moves
        // them down to their first use, where the warp would wait for them. (No instruction is emitted.)
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            asm volatile("" : "+f"(rq[e]), "+f"(rk[e]));
            if (MODE == 0) asm volatile("" : "+f"(rg[e]));
        }
        asm volatile("" : "+f"(rv), "+f"(r1), "+f"(r2));
    };
    auto stage = [&]() {
#pragma unroll
        for (int e = 0; e < PER; ++e) {
            const int idx = threadIdx.x + 128 * e, t = idx / DPAD, d = idx % DPAD;
            const int at = (d / DS) * SL + d % DS;
            const bool in = d < D;                     // channels beyond D stay out of every sum
            sq[t][at] = in ? (MODE == 1 ? rq[e] * p.q_scale : rq[e]) : 0.f;
            sk[t][at] = in ? rk[e] : 0.f;
            if (MODE == 0 && !head_decay) sg[t][at] = p.decay_ready ? rg[e] : expf(-a_rate * softplus_f(rg[e] + bias[e]));
        }
        if (threadIdx.x < SCAN_TOKENS * SCAN_COLS) {
            const int cc = blockIdx.z * SCAN_COLS + threadIdx.x % SCAN_COLS;
            sv[threadIdx.x / SCAN_COLS][threadIdx.x % SCAN_COLS] = cc < Dv ? rv : ((MODE == 1 && cc == Dv) ? 1.0f : 0.f);   // the column of n has v = 1
        }
        if (threadIdx.x < SCAN_TOKENS) {
            if (MODE == 0) {
                s1[threadIdx.x] = sigmoid_f(r1);
                if (head_decay) s2[threadIdx.x] = p.decay_ready ? r2 : expf(-a_rate * softplus_f(r2 + p.vec_b[hd]));
            } else if (MODE == 1) {
                s1[threadIdx.x] = p.cap * tanhf((r1 + p.vec_a[hd]) / p.cap);
                s2[threadIdx.x] = logsigmoid_f(p.cap * tanhf((r2 + p.vec_b[hd]) / p.cap));
            } else if (MODE == 3) { s1[threadIdx.x] = r1; s2[threadIdx.x] = r2; }
        }
    };
    fetch(0);
    for (int t0 = 0; t0 < n; t0 += SCAN_TOKENS) {
        const int nt = min(SCAN_TOKENS, n - t0);
        __syncthreads();                               // the tokens before are done with the staged values
        stage();
        __syncthreads();
        if (MODE == 0) {
            // k . q of every staged token, the same for all columns: warp w takes tokens 2w and 2w + 1
#pragma unroll
            for (int tt = 0; tt < SCAN_TOKENS / 4; ++tt) {
                const int t = warp * (SCAN_TOKENS / 4) + tt;
                float a = 0.f;
                for (int d = lane; d < DPAD; d += 32) {
                    const int at = (d / DS) * SL + d % DS;
                    a = fmaf(sk[t][at], sq[t][at], a);
                }
                a = warp_sum(a);
                if (lane == 0) skq[t] = a;
            }
            __syncthreads();
        }
        if (t0 + SCAN_TOKENS < n) fetch(t0 + SCAN_TOKENS);
        // Gated delta rule, one token. With S' = diag(g) S both products S'^T k and S'^T q are taken at once (two
        // butterflies side by side), and since the state after the write is S' + k u^T, the read-out is
        // S'^T q + u (k . q): the only thing the next token waits for is the write itself.
        auto delta_token = [&](int t) {
            const float* kq = &sk[t][slice * SL];
            const float* qq = &sq[t][slice * SL];
            const float* gg = &sg[t][slice * SL];
            const float vcol = sv[t][wcol];
            float kr[DS];
            float d4[4] = {0.f, 0.f, 0.f, 0.f}, o4[4] = {0.f, 0.f, 0.f, 0.f};       // four chains each, always in this order
            if (head_decay) {
                const float gh = s2[t];
#pragma unroll
                for (int i = 0; i < DS; ++i) S[i] *= gh;
            } else {
#pragma unroll
                for (int i = 0; i < DS; i += 4) {
                    const float4 gv = *reinterpret_cast<const float4*>(gg + i);
                    S[i] *= gv.x; S[i + 1] *= gv.y; S[i + 2] *= gv.z; S[i + 3] *= gv.w;
                }
            }
#pragma unroll
            for (int i = 0; i < DS; i += 4) {
                const float4 kv = *reinterpret_cast<const float4*>(kq + i);
                const float4 qv = *reinterpret_cast<const float4*>(qq + i);
                kr[i] = kv.x; kr[i + 1] = kv.y; kr[i + 2] = kv.z; kr[i + 3] = kv.w;
                d4[0] = fmaf(S[i], kv.x, d4[0]); d4[1] = fmaf(S[i + 1], kv.y, d4[1]);
                d4[2] = fmaf(S[i + 2], kv.z, d4[2]); d4[3] = fmaf(S[i + 3], kv.w, d4[3]);
                o4[0] = fmaf(S[i], qv.x, o4[0]); o4[1] = fmaf(S[i + 1], qv.y, o4[1]);
                o4[2] = fmaf(S[i + 2], qv.z, o4[2]); o4[3] = fmaf(S[i + 3], qv.w, o4[3]);
            }
            float dk = (d4[0] + d4[1]) + (d4[2] + d4[3]), dq = (o4[0] + o4[1]) + (o4[2] + o4[3]);
#pragma unroll
            for (int sh = 1; sh < NS; sh <<= 1) {
                const float a = __shfl_xor_sync(0xffffffffu, dk, sh), b = __shfl_xor_sync(0xffffffffu, dq, sh);
                dk += a;
                dq += b;
            }
            const float u = s1[t] * (vcol - dk);
#pragma unroll
            for (int i = 0; i < DS; ++i) S[i] = fmaf(kr[i], u, S[i]);
            if (live && slice == 0) p.out[(size_t)(row0 + t0 + t) * heads * Dv + hd * Dv + c] = fmaf(u, skq[t], dq);
        };
        if constexpr (MODE == 0) {
            if (nt == SCAN_TOKENS) {        // a whole round unrolled: the next tokens' loads and this one's read-out overlap
#pragma unroll
                for (int t = 0; t < SCAN_TOKENS; ++t) delta_token(t);
            } else {
                for (int t = 0; t < nt; ++t) delta_token(t);
            }
        } else if constexpr (MODE == 2 || MODE == 3) {
            // Retention, one token: S = d S + k v, then the read-out from the new state; four chains, always in this order.
            // The state-space recurrence is the same with a decay and a step of the token's own, and D v beside the read-out.
            auto retention_token = [&](int t) {
                const float* kq = &sk[t][slice * SL];
                const float* qq = &sq[t][slice * SL];
                const float raw = sv[t][wcol];
                const float vcol = MODE == 3 ? raw * s1[t] : raw, fade = MODE == 3 ? s2[t] : keep;
                float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int i = 0; i < DS; i += 4) {
                    const float4 kv = *reinterpret_cast<const float4*>(kq + i), qv = *reinterpret_cast<const float4*>(qq + i);
                    S[i] = fmaf(fade, S[i], vcol * kv.x); S[i + 1] = fmaf(fade, S[i + 1], vcol * kv.y);
                    S[i + 2] = fmaf(fade, S[i + 2], vcol * kv.z); S[i + 3] = fmaf(fade, S[i + 3], vcol * kv.w);
                    o4[0] = fmaf(S[i], qv.x, o4[0]); o4[1] = fmaf(S[i + 1], qv.y, o4[1]);
                    o4[2] = fmaf(S[i + 2], qv.z, o4[2]); o4[3] = fmaf(S[i + 3], qv.w, o4[3]);
                }
                float o = slices_sum<NS>((o4[0] + o4[1]) + (o4[2] + o4[3]));
                if (MODE == 3) o = fmaf(keep, raw, o);
                if (live && slice == 0) p.out[(size_t)(row0 + t0 + t) * heads * Dv + hd * Dv + c] = o;
            };
            if (nt == SCAN_TOKENS) {
#pragma unroll
                for (int t = 0; t < SCAN_TOKENS; ++t) retention_token(t);
            } else {
                for (int t = 0; t < nt; ++t) retention_token(t);
            }
        } else {
            for (int t = 0; t < nt; ++t) {
                const float* kq = &sk[t][slice * SL];
                const float* qq = &sq[t][slice * SL];
                const float vcol = sv[t][wcol];
                float o = 0.f;
                const float fm = s2[t] + m;
                const float m_new = fmaxf(fm, s1[t]);
                const float a = expf(fm - m_new);
                const float bv = expf(s1[t] - m_new) * vcol;
                m = m_new;
                float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int i = 0; i < DS; i += 4) {
                    const float4 kv = *reinterpret_cast<const float4*>(kq + i), qv = *reinterpret_cast<const float4*>(qq + i);
                    S[i] = fmaf(a, S[i], bv * kv.x); S[i + 1] = fmaf(a, S[i + 1], bv * kv.y);
                    S[i + 2] = fmaf(a, S[i + 2], bv * kv.z); S[i + 3] = fmaf(a, S[i + 3], bv * kv.w);
                    o4[0] = fmaf(S[i], qv.x, o4[0]); o4[1] = fmaf(S[i + 1], qv.y, o4[1]);
                    o4[2] = fmaf(S[i + 2], qv.z, o4[2]); o4[3] = fmaf(S[i + 3], qv.w, o4[3]);
                }
                o = slices_sum<NS>((o4[0] + o4[1]) + (o4[2] + o4[3]));
                if (live && slice == 0) {
                    float* orow = p.out + ((size_t)(row0 + t0 + t) * heads + hd) * (Dv + 2);
                    orow[c] = o;
                    if (c == Dv) orow[Dv + 1] = m;
                }
            }
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < DS; i += 4) {
            if (vec && d0 + i < D) {
                *reinterpret_cast<float4*>(st + d0 + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (d0 + i + j < D) st[d0 + i + j] = S[i + j];
            }
        }
        if (MODE == 1 && slice == 0) p.state_m[cell] = m;
    }
}

// Eight slices per column: with 16 or 32 (more and lighter warps for a lone prompt) the staging of q and k, which every
// block repeats, weighs as much as the shorter sums save, and a prompt ran no faster.
#define SCAN_SLICES 8

template <int MODE>
static int launch_scan(const ScanParams& p, int n_seqs, cudaStream_t s) {
    if (n_seqs <= 0) return 0;
    if (p.D < 1 || p.D > 256 || p.Dv < 1) return CML_ERR_BAD_SIZE;
    const int cols = MODE == 1 ? p.Dv + 1 : p.Dv;
    constexpr int block_cols = 128 / SCAN_SLICES;
    dim3 grid(n_seqs, p.heads, (cols + block_cols - 1) / block_cols);
#define SCAN_CASE(DS_)                                                                    \
    if (p.D <= SCAN_SLICES * DS_) {                                                       \
        launch_pdl(scan_kernel<DS_, MODE, SCAN_SLICES>, grid, dim3(128), 0, s, p);        \
        return cml_launch_status();                                                       \
    }
    SCAN_CASE(4) SCAN_CASE(8) SCAN_CASE(16) SCAN_CASE(32)
#undef SCAN_CASE
    return CML_ERR_BAD_SIZE;
}

extern "C" int cml_delta_scan(const float* qkv, long ldq, const float* beta_in, long ldb, int beta_col, const float* decay_in,
                              long ldd, const float* a_log, const float* dt_bias, float* state, const int* seq_row0,
                              const int* seq_new, const int* seq_start, const int* seq_slot, float* out, int n_seqs, int heads,
                              int qk_heads, int D, int Dv, int decay_ready, int decay_dim, void* stream) {
    if (qk_heads < 1 || heads % qk_heads || (decay_dim != 1 && decay_dim != D)) return CML_ERR_BAD_SIZE;
    ScanParams p = {};
    p.in_a = qkv; p.lda = ldq; p.in_b = beta_in; p.ldb = ldb; p.b_col = beta_col; p.in_c = decay_in; p.ldc = ldd;
    p.vec_a = a_log; p.vec_b = dt_bias; p.state = state; p.state_m = nullptr;
    p.seq_row0 = seq_row0; p.seq_new = seq_new; p.seq_start = seq_start; p.seq_slot = seq_slot; p.out = out;
    p.heads = heads; p.qk_heads = qk_heads; p.D = D; p.Dv = Dv; p.decay_ready = decay_ready; p.decay_dim = decay_dim;
    return launch_scan<0>(p, n_seqs, (cudaStream_t)stream);
}

extern "C" int cml_memory_scan(const float* proj, long ld, int q_col, int k_col, int v_col, int i_col, int f_col,
                               const float* i_bias, const float* f_bias, float cap, float q_scale, float* state,
                               float* state_m, const int* seq_row0, const int* seq_new, const int* seq_start,
                               const int* seq_slot, float* out, int n_seqs, int heads, int D, int Dv, void* stream) {
    ScanParams p = {};
    p.in_a = proj; p.lda = ld; p.vec_a = i_bias; p.vec_b = f_bias; p.state = state; p.state_m = state_m;
    p.seq_row0 = seq_row0; p.seq_new = seq_new; p.seq_start = seq_start; p.seq_slot = seq_slot; p.out = out;
    p.heads = heads; p.qk_heads = heads; p.D = D; p.Dv = Dv;
    p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.i_col = i_col; p.f_col = f_col; p.cap = cap; p.q_scale = q_scale;
    return launch_scan<1>(p, n_seqs, (cudaStream_t)stream);
}

extern "C" int cml_retention_scan(const float* proj, long ld, int q_col, int k_col, int v_col, const float* decay, float* state,
                                  const int* seq_row0, const int* seq_new, const int* seq_start, const int* seq_slot,
                                  float* out, int n_seqs, int heads, int D, int Dv, void* stream) {
    ScanParams p = {};
    p.in_a = proj; p.lda = ld; p.vec_a = decay; p.state = state; p.state_m = nullptr;
    p.seq_row0 = seq_row0; p.seq_new = seq_new; p.seq_start = seq_start; p.seq_slot = seq_slot; p.out = out;
    p.heads = heads; p.qk_heads = heads; p.D = D; p.Dv = Dv;
    p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.q_scale = 1.0f;
    return launch_scan<2>(p, n_seqs, (cudaStream_t)stream);
}

extern "C" int cml_ssm_scan(const float* rows_in, long ld, int x_col, int b_col, int c_col, const float* gates, long ldg,
                            const float* d_skip, float* state, const int* seq_row0, const int* seq_new, const int* seq_start,
                            const int* seq_slot, float* out, int n_seqs, int heads, int groups, int D, int Dv, void* stream) {
    if (groups < 1 || heads % groups) return CML_ERR_BAD_SIZE;
    ScanParams p = {};
    p.in_a = rows_in; p.lda = ld; p.in_b = gates; p.ldb = ldg; p.vec_a = d_skip; p.state = state; p.state_m = nullptr;
    p.seq_row0 = seq_row0; p.seq_new = seq_new; p.seq_start = seq_start; p.seq_slot = seq_slot; p.out = out;
    p.heads = heads; p.qk_heads = groups; p.D = D; p.Dv = Dv;
    p.q_col = c_col; p.k_col = b_col; p.v_col = x_col; p.q_scale = 1.0f;
    return launch_scan<3>(p, n_seqs, (cudaStream_t)stream);
}

// ------------------------------------------------------------------------------------
// What the state-space recurrence reads. proj [rows, ld] (n_splits matrices split_stride apart, added in split order):
// z (inner), then the convolved channels (x, B, C), then one step-size input per head. Every channel passes a causal
// convolution (conv_w [taps, channels], the last tap the current token's; `state` [slots, max(taps - 1, 1), channels] holds
// the inputs of the tokens before the step) with bias, then SiLU: out [rows, channels]. The steps: dt = softplus(in +
// dt_bias), gates [rows, 2 heads] = dt, then exp(-exp(a_log) dt). z_out (may be null) gets z [rows, inner]. With
// update_state (every sequence of the step brings one row) the state moves on by that row here. A thread takes VEC
// neighbouring columns of up to `rows_per` rows.
struct SsmInputs {
    const float* proj; long ld; int n_splits; long split_stride;
    const float* conv_w; const float* conv_b; const float* dt_bias; const float* a_log;
    float* state; int update_state;
    const int* row_seq; const int* row_pos; const int* seq_row0; const int* seq_slot;
    float* out; float* gates; float* z_out;
    int rows, rows_per, inner, channels, heads, taps;
};

template <int VEC> struct SsmPiece { float v[VEC]; };
template <int VEC> __device__ __forceinline__ SsmPiece<VEC> ssm_load(const float* p) {
    SsmPiece<VEC> r;
    if constexpr (VEC == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
    } else {
        r.v[0] = p[0];
    }
    return r;
}
template <int VEC> __device__ __forceinline__ void ssm_store(float* p, const SsmPiece<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else p[0] = r.v[0];
}
template <int VEC> __device__ __forceinline__ SsmPiece<VEC> ssm_sum(const float* p, int n, long stride) {
    SsmPiece<VEC> r = ssm_load<VEC>(p);
    for (int s0 = 1; s0 < n; s0 += 8) {                        // eight splits' loads in flight, added in split order
        SsmPiece<VEC> t[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) t[k] = ssm_load<VEC>(p + (size_t)min(s0 + k, n - 1) * stride);
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (s0 + k < n)
#pragma unroll
                for (int e = 0; e < VEC; ++e) r.v[e] += t[k].v[e];
    }
    return r;
}

template <int VEC>
__global__ void __launch_bounds__(128) ssm_inputs_kernel(const SsmInputs p) {
    pdl_wait();
    pdl_launch_dependents();
    const int nz = p.z_out ? p.inner / VEC : 0, nc = p.channels / VEC;
    const int u = blockIdx.x * blockDim.x + threadIdx.x;
    const int r0 = blockIdx.y * p.rows_per, r1 = min(p.rows, r0 + p.rows_per);
    if (u >= nc + nz) {                                        // a head's steps and decays
        const int h = u - nc - nz;
        if (h >= p.heads) return;
        const float bias = p.dt_bias[h], rate = expf(p.a_log[h]);
        for (int r = r0; r < r1; ++r) {
            const float dt = softplus_f(split_sum(p.proj + (size_t)r * p.ld + p.inner + p.channels + h, p.n_splits, p.split_stride) + bias);
            p.gates[(size_t)r * 2 * p.heads + h] = dt;
            p.gates[(size_t)r * 2 * p.heads + p.heads + h] = expf(-rate * dt);
        }
        return;
    }
    if (u >= nc) {                                             // z
        const int c = (u - nc) * VEC;
        for (int r = r0; r < r1; ++r)
            ssm_store<VEC>(p.z_out + (size_t)r * p.inner + c, ssm_sum<VEC>(p.proj + (size_t)r * p.ld + c, p.n_splits, p.split_stride));
        return;
    }
    const int c = u * VEC, taps = p.taps, keep = max(taps - 1, 1);
    const float* col = p.proj + p.inner + c;
    const SsmPiece<VEC> bias = ssm_load<VEC>(p.conv_b + c);
    SsmPiece<VEC> w[4];                                        // the taps of the token and of the three before it
#pragma unroll
    for (int back = 0; back < 4; ++back) w[back] = ssm_load<VEC>(p.conv_w + (size_t)max(taps - 1 - back, 0) * p.channels + c);
    for (int r = r0; r < r1; ++r) {
        const int s = p.row_seq[r], pos = p.row_pos[r], inside = r - p.seq_row0[s];
        float* st = p.state + (size_t)p.seq_slot[s] * keep * p.channels + c;
        auto input = [&](int back) -> SsmPiece<VEC> {
            return back <= inside ? ssm_sum<VEC>(col + (size_t)(r - back) * p.ld, p.n_splits, p.split_stride)
                                  : ssm_load<VEC>(st + (size_t)(taps - 1 + inside - back) * p.channels);
        };
        SsmPiece<VEC> acc = bias, own = input(0), before[3];
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            const bool there = k + 1 < taps && k + 1 <= pos;   // (a token before the sequence's start counts as zero)
            before[k] = there ? input(k + 1) : own;
            if (!there)
#pragma unroll
                for (int e = 0; e < VEC; ++e) before[k].v[e] = 0.f;
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e)
            acc.v[e] = fmaf(w[3].v[e], before[2].v[e], fmaf(w[2].v[e], before[1].v[e], fmaf(w[1].v[e], before[0].v[e], fmaf(w[0].v[e], own.v[e], acc.v[e]))));
        for (int back = 4; back < taps && back <= pos; ++back) {
            const SsmPiece<VEC> x = input(back), wb = ssm_load<VEC>(p.conv_w + (size_t)(taps - 1 - back) * p.channels + c);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc.v[e] = fmaf(wb.v[e], x.v[e], acc.v[e]);
        }
        if (p.update_state && taps > 1) {
            for (int j = 0; j + 2 < taps; ++j) {
                SsmPiece<VEC> t = ssm_load<VEC>(st + (size_t)(j + 1) * p.channels);
                if (pos + j + 2 < taps)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) t.v[e] = 0.f;
                ssm_store<VEC>(st + (size_t)j * p.channels, t);
            }
            ssm_store<VEC>(st + (size_t)(taps - 2) * p.channels, own);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc.v[e] = silu_f(acc.v[e]);
        ssm_store<VEC>(p.out + (size_t)r * p.channels + c, acc);
    }
}

// The same for prompts (complete rows, up to four taps): a thread asks for the inputs of SSI_ROWS neighbouring rows and of the three
// before them at once and keeps them in registers; what a row lacks within the step comes from the state.
#define SSI_ROWS 8
template <int VEC>
__global__ void __launch_bounds__(128) ssm_inputs_rows_kernel(const SsmInputs p) {
    pdl_wait();
    pdl_launch_dependents();
    const int nc = p.channels / VEC, u = blockIdx.x * blockDim.x + threadIdx.x;
    const int r0 = blockIdx.y * SSI_ROWS, r1 = min(p.rows, r0 + SSI_ROWS);
    if (u >= nc) {                                             // a head's steps and decays
        const int h = u - nc;
        if (h >= p.heads) return;
        const float bias = p.dt_bias[h], rate = expf(p.a_log[h]);
        float x[SSI_ROWS];
#pragma unroll
        for (int i = 0; i < SSI_ROWS; ++i) x[i] = p.proj[(size_t)min(r0 + i, p.rows - 1) * p.ld + p.inner + p.channels + h];
        for (int i = 0; i < r1 - r0; ++i) {
            float* o = p.gates + (size_t)(r0 + i) * 2 * p.heads + h;
            const float dt = softplus_f(x[i] + bias);
            o[0] = dt;
            o[p.heads] = expf(-rate * dt);
        }
        return;
    }
    const int c = u * VEC, taps = p.taps;
    const float* col = p.proj + p.inner + c;
    SsmPiece<VEC> x[SSI_ROWS + 3], w[4];
#pragma unroll
    for (int i = 0; i < SSI_ROWS + 3; ++i) x[i] = ssm_load<VEC>(col + (size_t)min(max(r0 + i - 3, 0), p.rows - 1) * p.ld);
    const SsmPiece<VEC> bias = ssm_load<VEC>(p.conv_b + c);
#pragma unroll
    for (int back = 0; back < 4; ++back) w[back] = ssm_load<VEC>(p.conv_w + (size_t)max(taps - 1 - back, 0) * p.channels + c);
#pragma unroll
    for (int i = 0; i < SSI_ROWS; ++i) {
        const int r = r0 + i;
        if (r >= r1) break;
        const int s = p.row_seq[r], pos = p.row_pos[r], inside = r - p.seq_row0[s];
        SsmPiece<VEC> acc = bias;
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc.v[e] = fmaf(w[0].v[e], x[i + 3].v[e], acc.v[e]);
#pragma unroll
        for (int back = 1; back < 4; ++back) {
            if (back >= taps || back > pos) break;             // (a token before the sequence's start counts as zero)
            SsmPiece<VEC> b = x[i + 3 - back];
            if (back > inside) b = ssm_load<VEC>(p.state + ((size_t)p.seq_slot[s] * (taps - 1) + taps - 1 + inside - back) * p.channels + c);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc.v[e] = fmaf(w[back].v[e], b.v[e], acc.v[e]);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc.v[e] = silu_f(acc.v[e]);
        ssm_store<VEC>(p.out + (size_t)r * p.channels + c, acc);
    }
}

extern "C" int cml_ssm_inputs(const float* proj, long ld, int n_splits, long split_stride, const float* conv_w, const float* conv_b,
                              const float* dt_bias, const float* a_log, float* state, int update_state, const int* row_seq,
                              const int* row_pos, const int* seq_row0, const int* seq_slot, float* out, float* gates, float* z_out,
                              int rows, int inner, int channels, int heads, int taps, void* stream) {
    if (rows <= 0) return 0;
    if (n_splits < 1 || inner < 1 || channels < 1 || heads < 1 || taps < 1) return CML_ERR_BAD_SIZE;
    SsmInputs p = {proj, ld, n_splits, split_stride, conv_w, conv_b, dt_bias, a_log, state, update_state, row_seq, row_pos, seq_row0,
                   seq_slot, out, gates, z_out, rows, 1, inner, channels, heads, taps};
    const bool vec = (((long)inner | (long)channels | ld | split_stride) & 3) == 0 &&
                     ((((uintptr_t)proj) | ((uintptr_t)conv_w) | ((uintptr_t)conv_b) | ((uintptr_t)state) | ((uintptr_t)out) | ((uintptr_t)z_out)) & 15) == 0;
    const int per = vec ? 4 : 1;
    const long units = (long)channels / per + (z_out ? inner / per : 0) + heads;
    if (!update_state && !z_out && n_splits == 1 && taps <= 4 && rows > 64 && rows <= 65535 * SSI_ROWS) {
        const dim3 grid((unsigned)((units + 127) / 128), (unsigned)((rows + SSI_ROWS - 1) / SSI_ROWS));
        if (vec) launch_pdl(ssm_inputs_rows_kernel<4>, grid, dim3(128), 0, (cudaStream_t)stream, p);
        else launch_pdl(ssm_inputs_rows_kernel<1>, grid, dim3(128), 0, (cudaStream_t)stream, p);
        return cml_launch_status();
    }
    if (((long)rows + p.rows_per - 1) / p.rows_per > 65535) p.rows_per = (int)((rows + 65534L) / 65535);
    const dim3 grid((unsigned)((units + 127) / 128), (unsigned)((rows + p.rows_per - 1) / p.rows_per));
    if (vec) launch_pdl(ssm_inputs_kernel<4>, grid, dim3(128), 0, (cudaStream_t)stream, p);
    else launch_pdl(ssm_inputs_kernel<1>, grid, dim3(128), 0, (cudaStream_t)stream, p);
    return cml_launch_status();
}

// After the state-space scan: v = y * silu(z), a row's `groups` equal parts each divided by its own root mean square
// (eps inside), times w, in the compute type. y [rows, width] float; z [rows, ldz] float; w [width] float; out rows ldo
// apart. A block owns one (row, part), whose values stay in shared memory between the two passes.
template <typename TO>
__global__ void __launch_bounds__(256) gated_group_norm_kernel(const float* __restrict__ y, const float* __restrict__ z, long ldz,
                                                               const float* __restrict__ w, TO* __restrict__ out, long ldo, int width,
                                                               int part, float eps) {
    extern __shared__ __align__(16) float gg_row[];
    __shared__ float red[32];
    pdl_wait();
    pdl_launch_dependents();
    const int r = blockIdx.x, c0 = blockIdx.y * part;
    const float* yr = y + (size_t)r * width + c0;
    const float* zr = z + (size_t)r * ldz + c0;
    float ss = 0.f;
    const bool vec = (((long)part | (long)width | ldz) & 3) == 0 && ((((uintptr_t)y) | ((uintptr_t)z)) & 15) == 0;
    if (vec) {
        for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4) {
            const float4 a = *reinterpret_cast<const float4*>(yr + c), g = *reinterpret_cast<const float4*>(zr + c);
            const float4 v = make_float4(a.x * silu_f(g.x), a.y * silu_f(g.y), a.z * silu_f(g.z), a.w * silu_f(g.w));
            *reinterpret_cast<float4*>(gg_row + c) = v;
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
    } else {
        for (int c = threadIdx.x; c < part; c += blockDim.x) {
            const float v = yr[c] * silu_f(zr[c]);
            gg_row[c] = v;
            ss = fmaf(v, v, ss);
        }
    }
    const float scale = 1.0f / sqrtf(block_sum(ss, red) / (float)part + eps);
    TO* o = out + (size_t)r * ldo + c0;
    if (vec) {                                                 // each thread reads back what it wrote itself
        for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[c + e] = from_f32<TO>(gg_row[c + e] * scale * w[c0 + c + e]);
    } else {
        for (int c = threadIdx.x; c < part; c += blockDim.x) o[c] = from_f32<TO>(gg_row[c] * scale * w[c0 + c]);
    }
}

extern "C" int cml_gated_group_norm(const float* y, const float* z, long ldz, const float* w, void* out, long ldo, int out_dtype, int rows,
                                    int width, int groups, float eps, void* stream) {
    if (rows <= 0) return 0;
    if (groups < 1 || groups > 65535 || width % groups) return CML_ERR_BAD_SIZE;
    const int part = width / groups;
    const size_t smem = (size_t)part * sizeof(float);
    if (smem > 200 * 1024) return CML_ERR_BAD_SIZE;
    const int block = part >= 1024 ? 256 : part >= 256 ? 128 : part >= 64 ? 64 : 32;
#define GG_CASE(T_, D_)                                                                                                   \
    if (out_dtype == D_) {                                                                                                \
        if (smem > 48 * 1024 && cml_allow_smem<gated_group_norm_kernel<T_>>(smem) != cudaSuccess) return CML_ERR_BAD_SIZE; \
        launch_pdl(gated_group_norm_kernel<T_>, dim3(rows, groups), dim3(block), smem, (cudaStream_t)stream, y, z, ldz, w, \
                   (T_*)out, ldo, width, part, eps);                                                                      \
        return cml_launch_status();                                                                                       \
    }
    GG_CASE(float, CML_DTYPE_F32)
    GG_CASE(bf16, CML_DTYPE_BF16)
#undef GG_CASE
    return CML_ERR_BAD_DTYPE;
}

// ------------------------------------------------------------------------------------
// Generalized delta rule. Both terms of the write read the old state, so with p = k^T S (S before the token), q = (r * w)^T S,
// n2 = 1 / (sum k^2 + 1e-6) the token is
//
//   S' = diag(w) S + k (v - a * (n2 p))^T,     o = q - n2 (sum r a k) p + (sum r k) v
//
// and the two products over the state, p and q, are taken side by side. What does not depend on the state is made
// beforehand, once per (row, head), by the kernel below: `packed` [rows, heads, 4 D + Dv] = k, r * w, w, a, v and `scal`
// [rows, heads, 4] = n2, n2 sum r a k, sum r k, 0.
//
// proj (n_splits matrices split_stride apart, added in split order) [rows, ld]: columns r, k (heads x D each), v
// (heads x Dv), the removal rates' inputs (heads x D), the gate's (heads x Dv), then `rank` columns of the decays' narrow
// inputs. a = sigmoid(in + a_bias). The decays' inputs z come as a product of their own (`high`, n_high matrices
// high_stride apart [rows, heads x D]) or, where `high` is null, are made here: z = W2 tanh(narrow), W2 [heads x D, rank].
// w = exp(-rate * sigmoid(z + w0)). gate_out (may be null) gets the gate's summed inputs [rows, heads x Dv].
struct DeltaInputs {
    const float* proj; long ld; int n_splits; long split_stride;
    const float* high; int n_high; long high_stride;
    const void* w2; int rank;
    const float* a_bias; const float* w0;
    float rate;
    float* packed; float* scal; float* gate_out;
    int heads, D, Dv;
};

template <typename T>
__global__ void __launch_bounds__(256) delta_inputs_kernel(const DeltaInputs p) {
    extern __shared__ __align__(16) float di_low[];            // tanh of the narrow inputs
    __shared__ float red0[32], red1[32], red2[32];
    pdl_wait();
    pdl_launch_dependents();
    const int r = blockIdx.x, hd = blockIdx.y, D = p.D, Dv = p.Dv, HD = p.heads * p.D, HV = p.heads * p.Dv;
    const float* row = p.proj + (size_t)r * p.ld;
    if (p.high == nullptr) {
        const float* narrow = row + 3 * HD + 2 * HV;
        for (int j = threadIdx.x; j < p.rank; j += blockDim.x) di_low[j] = tanhf(split_sum(narrow + j, p.n_splits, p.split_stride));
        __syncthreads();
    }
    float* pk = p.packed + ((size_t)r * p.heads + hd) * (4 * D + Dv);
    float k2 = 0.f, rak = 0.f, rk = 0.f;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        const int c = hd * D + d;
        const float rr = split_sum(row + c, p.n_splits, p.split_stride);
        const float kk = split_sum(row + HD + c, p.n_splits, p.split_stride);
        const float aa = sigmoid_f(split_sum(row + 2 * HD + HV + c, p.n_splits, p.split_stride) + p.a_bias[c]);
        float z = 0.f;
        if (p.high != nullptr) {
            z = split_sum(p.high + (size_t)r * HD + c, p.n_high, p.high_stride);
        } else {
            const T* w = (const T*)p.w2 + (size_t)c * p.rank;
            constexpr int PIECE = 16 / (int)sizeof(T);
            int j = 0;
            if (p.rank % PIECE == 0 && (((uintptr_t)p.w2) & 15) == 0) {
                for (; j < p.rank; j += PIECE) {
                    union { uint4 raw; T e[PIECE]; } v;
                    v.raw = *reinterpret_cast<const uint4*>(w + j);
#pragma unroll
                    for (int e = 0; e < PIECE; ++e) z = fmaf(to_f32(v.e[e]), di_low[j + e], z);
                }
            } else {
                for (; j < p.rank; ++j) z = fmaf(to_f32(w[j]), di_low[j], z);
            }
        }
        const float ww = expf(-p.rate * sigmoid_f(z + p.w0[c]));
        pk[d] = kk;
        pk[D + d] = rr * ww;
        pk[2 * D + d] = ww;
        pk[3 * D + d] = aa;
        k2 = fmaf(kk, kk, k2);
        rak = fmaf(rr * aa, kk, rak);
        rk = fmaf(rr, kk, rk);
    }
    for (int c = threadIdx.x; c < Dv; c += blockDim.x) {
        pk[4 * D + c] = split_sum(row + 2 * HD + hd * Dv + c, p.n_splits, p.split_stride);
        if (p.gate_out) p.gate_out[(size_t)r * HV + hd * Dv + c] = split_sum(row + 3 * HD + HV + hd * Dv + c, p.n_splits, p.split_stride);
    }
    k2 = block_sum(k2, red0);
    rak = block_sum(rak, red1);
    rk = block_sum(rk, red2);
    if (threadIdx.x == 0) {
        const float n2 = 1.0f / (k2 + 1e-6f);
        float4* out = reinterpret_cast<float4*>(p.scal + ((size_t)r * p.heads + hd) * 4);
        *out = make_float4(n2, n2 * rak, rk, 0.f);
    }
}

extern "C" int cml_delta_inputs(const float* proj, long ld, int n_splits, long split_stride, const float* high, int n_high,
                                long high_stride, const void* w2, int dtype, int rank, const float* a_bias, const float* w0,
                                float rate, float* packed, float* scal, float* gate_out, int rows, int heads, int D, int Dv,
                                void* stream) {
    if (rows <= 0) return 0;
    if (heads < 1 || heads > 65535 || D < 1 || Dv < 1 || n_splits < 1 || rank < 0 || rank > 8192) return CML_ERR_BAD_SIZE;
    if (high == nullptr ? w2 == nullptr : n_high < 1) return CML_ERR_BAD_SIZE;
    if (((uintptr_t)scal) & 15) return CML_ERR_BAD_ALIGN;
    DeltaInputs p = {proj, ld, n_splits, split_stride, high, n_high, high_stride, w2, rank, a_bias, w0, rate, packed, scal, gate_out,
                     heads, D, Dv};
    const int most = D > Dv ? D : Dv;
    const int block = most >= 256 ? 256 : (most + 31) / 32 * 32;
    const size_t smem = high == nullptr ? (size_t)rank * sizeof(float) : 0;
    if (dtype == CML_DTYPE_F32)
        launch_pdl(delta_inputs_kernel<float>, dim3(rows, heads), dim3(block), smem, (cudaStream_t)stream, p);
    else if (dtype == CML_DTYPE_BF16)
        launch_pdl(delta_inputs_kernel<bf16>, dim3(rows, heads), dim3(block), smem, (cudaStream_t)stream, p);
    else
        return CML_ERR_BAD_DTYPE;
    return cml_launch_status();
}

// The scan: like the scans above a block of 128 threads owns 128 / NS columns of one (sequence, head), NS threads of a warp
// share a column (a slice of DS key channels each) and walk the new tokens in order. The prepared rows of
// GD_TOKENS tokens come by cp.async into one of two buffers of shared memory while the other one's are worked on.
#define GD_TOKENS 8
struct GeneralDelta {
    const float* packed; const float* scal; float* state;
    const int* seq_row0; const int* seq_new; const int* seq_start; const int* seq_slot;
    float* out;
    int heads, D, Dv;
};

template <int BYTES>
__device__ __forceinline__ void gd_copy(float* smem, const float* gmem) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
    if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(s), "l"(gmem) : "memory");
}

template <int DS, int NS>
__global__ void __launch_bounds__(128) general_delta_kernel(const GeneralDelta p) {
    constexpr int COLS = 128 / NS;
    constexpr int SL = DS == 4 ? 4 : DS + 4;               // floats of a slice in shared memory (padded against bank conflicts)
    constexpr int ROW = NS * SL;                           // floats of one array of a token
    constexpr int TOKEN = 4 * ROW + COLS + 4;              // k, r * w, w, a; the block's values; the scalars
    extern __shared__ __align__(16) float gd_sh[];         // [2][GD_TOKENS][TOKEN]
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, hd = blockIdx.y;
    const int D = p.D, Dv = p.Dv, heads = p.heads;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, slice = lane % NS;
    const int wcol = warp * (32 / NS) + lane / NS;
    const int col0 = blockIdx.z * COLS, c = col0 + wcol;
    const bool live = c < Dv;
    const int d0 = slice * DS;
    const int row0 = p.seq_row0[s], n = p.seq_new[s];
    const bool fresh = p.seq_start[s] == 0, vec = ((D | Dv) & 3) == 0;     // whole heads of `packed` start on 16 bytes
    const size_t per_head = 4 * D + Dv, per_row = per_head * heads;
    float* st = p.state + (((size_t)p.seq_slot[s] * heads + hd) * Dv + (live ? c : 0)) * D;
    auto fetch = [&](int t0, int buf) {
        const int nt = min(GD_TOKENS, n - t0);
        float* dst = gd_sh + (size_t)buf * GD_TOKENS * TOKEN;
        const float* src = p.packed + (size_t)(row0 + t0) * per_row + (size_t)hd * per_head;
        if (vec) {
            const int q = D / 4;                           // 16-byte pieces of an array; a warp takes every fourth (token, array)
            for (int ta = warp; ta < 4 * nt; ta += 4)
                for (int i = lane; i < q; i += 32) {
                    const int d = 4 * i;
                    gd_copy<16>(dst + (ta >> 2) * TOKEN + (ta & 3) * ROW + (d / DS) * SL + d % DS, src + (size_t)(ta >> 2) * per_row + (ta & 3) * D + d);
                }
        } else {
            for (int ta = warp; ta < 4 * nt; ta += 4)
                for (int d = lane; d < D; d += 32)
                    gd_copy<4>(dst + (ta >> 2) * TOKEN + (ta & 3) * ROW + (d / DS) * SL + d % DS, src + (size_t)(ta >> 2) * per_row + (ta & 3) * D + d);
        }
        for (int i = threadIdx.x; i < nt * COLS; i += 128) {
            const int t = i / COLS, cc = i % COLS;
            if (col0 + cc < Dv) gd_copy<4>(dst + t * TOKEN + 4 * ROW + cc, src + (size_t)t * per_row + 4 * D + col0 + cc);
        }
        if (threadIdx.x < nt)
            gd_copy<16>(dst + threadIdx.x * TOKEN + 4 * ROW + COLS, p.scal + ((size_t)(row0 + t0 + threadIdx.x) * heads + hd) * 4);
    };
    if (D < NS * DS || Dv - col0 < COLS) {                 // channels and columns that are not there stay zero
        for (int i = threadIdx.x; i < 2 * GD_TOKENS * TOKEN; i += 128) gd_sh[i] = 0.f;
        __syncthreads();
    }
    fetch(0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    float S[DS];
#pragma unroll
    for (int i = 0; i < DS; i += 4) {
        if (live && !fresh && vec && d0 + i < D) {
            const float4 t = *reinterpret_cast<const float4*>(st + d0 + i);
            S[i] = t.x; S[i + 1] = t.y; S[i + 2] = t.z; S[i + 3] = t.w;
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) S[i + j] = (live && !fresh && d0 + i + j < D) ? st[d0 + i + j] : 0.f;
        }
    }
    for (int t0 = 0, buf = 0; t0 < n; t0 += GD_TOKENS, buf ^= 1) {
        if (t0 + GD_TOKENS < n) fetch(t0 + GD_TOKENS, buf ^ 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");           // all but the newest group: this round's tokens are here
        __syncthreads();
        const float* base = gd_sh + (size_t)buf * GD_TOKENS * TOKEN;
        auto token = [&](int t) {
            const float* tk = base + t * TOKEN + slice * SL;
            const float vcol = base[t * TOKEN + 4 * ROW + wcol];
            const float4 sc = *reinterpret_cast<const float4*>(base + t * TOKEN + 4 * ROW + COLS);
            float kr[DS], p4[4] = {0.f, 0.f, 0.f, 0.f}, q4[4] = {0.f, 0.f, 0.f, 0.f};      // four chains each, always in this order
#pragma unroll
            for (int i = 0; i < DS; i += 4) {
                const float4 kv = *reinterpret_cast<const float4*>(tk + i), rv = *reinterpret_cast<const float4*>(tk + ROW + i);
                kr[i] = kv.x; kr[i + 1] = kv.y; kr[i + 2] = kv.z; kr[i + 3] = kv.w;
                p4[0] = fmaf(S[i], kv.x, p4[0]); p4[1] = fmaf(S[i + 1], kv.y, p4[1]);
                p4[2] = fmaf(S[i + 2], kv.z, p4[2]); p4[3] = fmaf(S[i + 3], kv.w, p4[3]);
                q4[0] = fmaf(S[i], rv.x, q4[0]); q4[1] = fmaf(S[i + 1], rv.y, q4[1]);
                q4[2] = fmaf(S[i + 2], rv.z, q4[2]); q4[3] = fmaf(S[i + 3], rv.w, q4[3]);
            }
            float pk = (p4[0] + p4[1]) + (p4[2] + p4[3]), qr = (q4[0] + q4[1]) + (q4[2] + q4[3]);
#pragma unroll
            for (int sh = 1; sh < NS; sh <<= 1) {
                const float x = __shfl_xor_sync(0xffffffffu, pk, sh), y = __shfl_xor_sync(0xffffffffu, qr, sh);
                pk += x;
                qr += y;
            }
            const float rem = -sc.x * pk;
#pragma unroll
            for (int i = 0; i < DS; i += 4) {
                const float4 wv = *reinterpret_cast<const float4*>(tk + 2 * ROW + i), av = *reinterpret_cast<const float4*>(tk + 3 * ROW + i);
                S[i] = fmaf(kr[i], fmaf(av.x, rem, vcol), wv.x * S[i]);
                S[i + 1] = fmaf(kr[i + 1], fmaf(av.y, rem, vcol), wv.y * S[i + 1]);
                S[i + 2] = fmaf(kr[i + 2], fmaf(av.z, rem, vcol), wv.z * S[i + 2]);
                S[i + 3] = fmaf(kr[i + 3], fmaf(av.w, rem, vcol), wv.w * S[i + 3]);
            }
            // (a plain store might alias the buffers in shared memory as far as the compiler knows, and hold back the next token's loads)
            if (live && slice == 0)
                asm volatile("st.global.f32 [%0], %1;" ::"l"(p.out + ((size_t)(row0 + t0 + t) * heads + hd) * Dv + c), "f"(fmaf(sc.z, vcol, fmaf(-sc.y, pk, qr))));
        };
        const int nt = min(GD_TOKENS, n - t0);
        if (nt == GD_TOKENS) {                             // a whole round unrolled: the next tokens' loads and this one's read-out overlap
#pragma unroll
            for (int t = 0; t < GD_TOKENS; ++t) token(t);
        } else {
            for (int t = 0; t < nt; ++t) token(t);
        }
        __syncthreads();                                   // before the next fetch overwrites this buffer
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < DS; i += 4) {
            if (vec && d0 + i < D) {
                *reinterpret_cast<float4*>(st + d0 + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (d0 + i + j < D) st[d0 + i + j] = S[i + j];
            }
        }
    }
}

extern "C" int cml_general_delta_scan(const float* packed, const float* scal, float* state, const int* seq_row0, const int* seq_new,
                                      const int* seq_start, const int* seq_slot, float* out, int n_seqs, int heads, int D, int Dv,
                                      void* stream) {
    if (n_seqs <= 0) return 0;
    if (D < 1 || D > 256 || Dv < 1 || heads < 1 || heads > 65535) return CML_ERR_BAD_SIZE;
    if ((((uintptr_t)packed) | ((uintptr_t)scal) | ((uintptr_t)state)) & 15) return CML_ERR_BAD_ALIGN;
    GeneralDelta p = {packed, scal, state, seq_row0, seq_new, seq_start, seq_slot, out, heads, D, Dv};
    constexpr int NS = SCAN_SLICES, COLS = 128 / NS;
    dim3 grid(n_seqs, heads, (Dv + COLS - 1) / COLS);
#define GD_CASE(DS_)                                                                                                     \
    if (D <= NS * DS_) {                                                                                                 \
        constexpr size_t smem = (size_t)2 * GD_TOKENS * (4 * NS * (DS_ == 4 ? 4 : DS_ + 4) + COLS + 4) * sizeof(float);  \
        if (smem > 48 * 1024 && cml_allow_smem<general_delta_kernel<DS_, NS>>(smem) != cudaSuccess) return CML_ERR_BAD_SIZE; \
        launch_pdl(general_delta_kernel<DS_, NS>, grid, dim3(128), smem, (cudaStream_t)stream, p);                       \
        return cml_launch_status();                                                                                      \
    }
    GD_CASE(4) GD_CASE(8) GD_CASE(16) GD_CASE(32)
#undef GD_CASE
    return CML_ERR_BAD_SIZE;
}

// ------------------------------------------------------------------------------------
// The state-space recurrence by chunks of SSQ = 64 tokens, for steps that bring many tokens per sequence. With a = -exp(A_log) dt,
// c_t the sum of a over the chunk's tokens up to t and S the state before the chunk, a token of the chunk reads
//
//   y_t = e^(c_t) S^T C_t + sum over s <= t of e^(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//
// and the state after the chunk is e^(c_last) S + sum over s of e^(c_last - c_s) dt_s B_s x_s^T. Three kernels: the products
// C_t . B_s of every (chunk, group) and the steps of its heads side by side; the states, each block walking a sequence's chunks with a tile of one head's
// state in registers and leaving the state before every chunk; the outputs of every (chunk, head) side by side. All float (every
// exponent is at most 0). Tokens that a chunk does not have count as zero steps.
#define SSQ 64

struct SsmChunks {
    const float* rows; long ld; int x_col, b_col, c_col;       // x (heads x P), B, C (groups x N) of ssm_inputs_kernel
    const float* gates; long ldg;                              // dt at column head
    const float* a_log; const float* d_skip;
    const int* tile_seq; const int* tile_q0;                   // chunks: sequence and first of its new rows
    const int* seq_row0; const int* seq_new; const int* seq_start; const int* seq_slot;
    float* state;                                              // [slots, heads, P, N]
    float* scores;                                             // [chunks, groups, SSQ, SSQ]
    float* steps;                                              // [chunks, heads, 3, SSQ]: c_t, dt_t, e^(c_last - c_t) dt_t
    float* prev;                                               // [chunks, heads, P, N]: the state before the chunk
    float* out;                                                // [rows, heads x P]
    int heads, groups, N, P;
};

// two products and sums in one instruction, each rounded as by itself
__device__ __forceinline__ void ssm_fma2(unsigned long long& d, unsigned long long a, unsigned long long b) {
    asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(d) : "l"(a), "l"(b));
}
struct SsmQuad { unsigned long long lo, hi; };                 // four floats as two pairs
__device__ __forceinline__ SsmQuad ssm_quad(const float* p) {
    const ulonglong2 t = *reinterpret_cast<const ulonglong2*>(p);
    return {t.x, t.y};
}
__device__ __forceinline__ float ssm_pair_sum(unsigned long long v) { return __uint_as_float((unsigned)v) + __uint_as_float((unsigned)(v >> 32)); }

// rows [row0 + min(i, nt - 1)] of `cols` floats at column col into shared rows of `pitch` floats; cp.async, 16 bytes a copy
__device__ __forceinline__ void ssm_stage(float* dst, int pitch, const float* src, long ld, int nt, int cols, int tid, int threads) {
    const int q = cols / 4;
    for (int i = tid; i < SSQ * q; i += threads) {
        const int t = i / q, c = (i - t * q) * 4;
        gd_copy<16>(dst + t * pitch + c, src + (size_t)min(t, nt - 1) * ld + c);
    }
}

// 64 x 64 products of rows of A and rows of B over N channels: thread (ty, px) of 8 x 16 takes rows ty + 8 i of A and rows
// 16 j + px of B; even and odd channels are summed side by side and added at the end
__device__ __forceinline__ void ssm_dot_tile(const float* a, const float* b, int pitch, int N, int ty, int px, float (&out)[8][4]) {
    unsigned long long acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0ull;
    for (int n = 0; n < N; n += 4) {
        SsmQuad bq[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) bq[j] = ssm_quad(b + (16 * j + px) * pitch + n);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const SsmQuad aq = ssm_quad(a + (ty + 8 * i) * pitch + n);
#pragma unroll
            for (int j = 0; j < 4; ++j) { ssm_fma2(acc[i][j], aq.lo, bq[j].lo); ssm_fma2(acc[i][j], aq.hi, bq[j].hi); }
        }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) out[i][j] = ssm_pair_sum(acc[i][j]);
}

// a warp: the running sums c_t of a chunk's 64 tokens (two a lane), their steps, and what their B count in the state after the chunk
__device__ __forceinline__ void ssm_steps(const SsmChunks& p, int tile, int row, int nt, int hd, int lane) {
    const float rate = expf(p.a_log[hd]);
    float dt[2], c[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        const float v = p.gates[(size_t)(row + min(t, nt - 1)) * p.ldg + hd];
        dt[e] = t < nt ? v : 0.f;
    }
    c[0] = -rate * dt[0];
    c[1] = c[0] - rate * dt[1];
    float before = c[1];
#pragma unroll
    for (int sh = 1; sh < 32; sh <<= 1) {
        const float o = __shfl_up_sync(0xffffffffu, before, sh);
        if (lane >= sh) before += o;
    }
    before -= c[1];                                            // the sum before this lane's two tokens
    c[0] += before;
    c[1] += before;
    const float last = __shfl_sync(0xffffffffu, c[1], 31);
    float2* o = reinterpret_cast<float2*>(p.steps + ((size_t)tile * p.heads + hd) * 3 * SSQ) + lane;
    o[0] = make_float2(c[0], c[1]);
    o[SSQ / 2] = make_float2(dt[0], dt[1]);
    o[SSQ] = make_float2(dt[0] * expf(last - c[0]), dt[1] * expf(last - c[1]));
}

__global__ void __launch_bounds__(128, 3) ssm_scores_kernel(const SsmChunks p) {
    extern __shared__ __align__(16) float ss_sh[];
    pdl_wait();
    pdl_launch_dependents();
    const int tile = blockIdx.x, g = blockIdx.y, tid = threadIdx.x, N = p.N, pitch = N + 4;
    const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile], nt = min(SSQ, p.seq_new[seq] - q0);
    const float* base = p.rows + (size_t)(p.seq_row0[seq] + q0) * p.ld + g * N;
    float* sC = ss_sh;
    float* sB = sC + SSQ * pitch;
    ssm_stage(sC, pitch, base + p.c_col, p.ld, nt, N, tid, 128);
    ssm_stage(sB, pitch, base + p.b_col, p.ld, nt, N, tid, 128);
    const int per = p.heads / p.groups;                        // meanwhile the steps of the group's heads
    for (int h = tid >> 5; h < per; h += 4) ssm_steps(p, tile, p.seq_row0[seq] + q0, nt, g * per + h, tid & 31);
    asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int px = tid & 15, ty = tid >> 4;
    float acc[8][4];
    ssm_dot_tile(sC, sB, pitch, N, ty, px, acc);
    float* o = p.scores + ((size_t)tile * p.groups + g) * SSQ * SSQ;
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[(ty + 8 * i) * SSQ + 16 * j + px] = acc[i][j];
}

// A block of 128 threads owns 64 values x 32 channels of one (sequence, head)'s state, four by four a thread.
#define SST_P 64
#define SST_N 32
__global__ void __launch_bounds__(128) ssm_states_kernel(const SsmChunks p) {
    extern __shared__ __align__(16) float st_sh[];             // two buffers of x, B, the tokens' weights, c_t
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, hd = blockIdx.y, N = p.N, P = p.P, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int n_tiles_n = (N + SST_N - 1) / SST_N;
    const int p0 = (int)(blockIdx.z / n_tiles_n) * SST_P, n0 = (int)(blockIdx.z % n_tiles_n) * SST_N;
    const int g = hd / (p.heads / p.groups), row0 = p.seq_row0[s], n = p.seq_new[s], n_chunks = (n + SSQ - 1) / SSQ;
    const bool fresh = p.seq_start[s] == 0;
    constexpr int BUF = SSQ * (SST_P + SST_N + 2);
    int first = 0;                                             // chunks of the sequences before this one
    for (int q = 0; q < s; ++q) first += (p.seq_new[q] + SSQ - 1) / SSQ;
    const int pc = (warp * 4 + (lane >> 3)) * 4, nc = (lane & 7) * 4;          // this thread's values and channels within the tile
    const bool live_n = n0 + nc < N;
    float* st = p.state + ((size_t)p.seq_slot[s] * p.heads + hd) * P * N;
    float4 S[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const bool ok = live_n && p0 + pc + e < P && !fresh;
        S[e] = ok ? *reinterpret_cast<const float4*>(st + (size_t)(p0 + pc + e) * N + n0 + nc) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (P - p0 < SST_P || N - n0 < SST_N) {                    // values and channels that are not there stay zero
        for (int i = tid; i < 2 * BUF; i += 128) st_sh[i] = 0.f;
        __syncthreads();
    }
    const int wp = min(SST_P, P - p0), wn = min(SST_N, N - n0);
    auto fetch = [&](int ch, int buf) {
        const int nt = min(SSQ, n - ch * SSQ);
        const float* base = p.rows + (size_t)(row0 + ch * SSQ) * p.ld;
        const float* xs = base + p.x_col + hd * P + p0;
        const float* bs = base + p.b_col + g * N + n0;
        float* dst = st_sh + buf * BUF;
        if (wp == SST_P) {                                     // whole tiles: places known when compiled
#pragma unroll
            for (int i = 0; i < SSQ * SST_P / 512; ++i) {
                const int t = (tid >> 4) + 8 * i, c = (tid & 15) * 4;
                gd_copy<16>(dst + t * SST_P + c, xs + (size_t)min(t, nt - 1) * p.ld + c);
            }
        } else ssm_stage(dst, SST_P, xs, p.ld, nt, wp, tid, 128);
        if (wn == SST_N) {
#pragma unroll
            for (int i = 0; i < SSQ * SST_N / 512; ++i) {
                const int t = (tid >> 3) + 16 * i, c = (tid & 7) * 4;
                gd_copy<16>(dst + SSQ * SST_P + t * SST_N + c, bs + (size_t)min(t, nt - 1) * p.ld + c);
            }
        } else ssm_stage(dst + SSQ * SST_P, SST_N, bs, p.ld, nt, wn, tid, 128);
        // the tokens' weights, then c_t
        const float* steps = p.steps + ((size_t)(first + ch) * p.heads + hd) * 3 * SSQ;
        if (tid < 32) gd_copy<16>(dst + SSQ * (SST_P + SST_N) + tid * 4, steps + (tid < 16 ? 2 * SSQ + tid * 4 : (tid - 16) * 4));
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);
    for (int ch = 0; ch < n_chunks; ++ch) {
        const float* sx = st_sh + (ch & 1) * BUF;
        const float* sb = sx + SSQ * SST_P;
        const float* sw = sb + SSQ * SST_N;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                       // this chunk is here, the other buffer is free
        if (ch + 1 < n_chunks) fetch(ch + 1, (ch + 1) & 1);
        // the state before the chunk, for the outputs
        float* pv = p.prev + ((size_t)(first + ch) * p.heads + hd) * P * N;
        const float keep = expf(sw[2 * SSQ - 1]);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            if (live_n && p0 + pc + e < P) *reinterpret_cast<float4*>(pv + (size_t)(p0 + pc + e) * N + n0 + nc) = S[e];
            S[e].x *= keep; S[e].y *= keep; S[e].z *= keep; S[e].w *= keep;
        }
#pragma unroll 8
        for (int t = 0; t < SSQ; ++t) {
            const float w = sw[t];
            const float4 x = *reinterpret_cast<const float4*>(sx + t * SST_P + pc);
            float4 b = *reinterpret_cast<const float4*>(sb + t * SST_N + nc);
            b.x *= w; b.y *= w; b.z *= w; b.w *= w;
            S[0].x = fmaf(x.x, b.x, S[0].x); S[0].y = fmaf(x.x, b.y, S[0].y); S[0].z = fmaf(x.x, b.z, S[0].z); S[0].w = fmaf(x.x, b.w, S[0].w);
            S[1].x = fmaf(x.y, b.x, S[1].x); S[1].y = fmaf(x.y, b.y, S[1].y); S[1].z = fmaf(x.y, b.z, S[1].z); S[1].w = fmaf(x.y, b.w, S[1].w);
            S[2].x = fmaf(x.z, b.x, S[2].x); S[2].y = fmaf(x.z, b.y, S[2].y); S[2].z = fmaf(x.z, b.z, S[2].z); S[2].w = fmaf(x.z, b.w, S[2].w);
            S[3].x = fmaf(x.w, b.x, S[3].x); S[3].y = fmaf(x.w, b.y, S[3].y); S[3].z = fmaf(x.w, b.z, S[3].z); S[3].w = fmaf(x.w, b.w, S[3].w);
        }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e)
        if (live_n && p0 + pc + e < P) *reinterpret_cast<float4*>(st + (size_t)(p0 + pc + e) * N + n0 + nc) = S[e];
}

// One block per (chunk, head, 64 values): 64 tokens x 64 values, thread (ty, px) of 8 x 16 takes tokens ty + 8 i and values
// 4 px .. 4 px + 3. The state's rows lie in shared memory so that the rows 4 px + j of neighbouring threads are neighbours.
#define SSM_PITCH 68                                           // floats of a row of the weights and of x in shared memory
__global__ void __launch_bounds__(128, 3) ssm_outputs_kernel(const SsmChunks p) {
    extern __shared__ __align__(16) float so_sh[];
    __shared__ float s_dt[SSQ], s_c[SSQ];
    pdl_wait();
    pdl_launch_dependents();
    const int tile = blockIdx.x, hd = blockIdx.y, p0 = blockIdx.z * 64, tid = threadIdx.x, N = p.N, P = p.P, pitch = N + 4;
    const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile], nt = min(SSQ, p.seq_new[seq] - q0), row0 = p.seq_row0[seq] + q0;
    const int g = hd / (p.heads / p.groups), wp = min(64, P - p0);
    const float* base = p.rows + (size_t)row0 * p.ld;
    const int area = SSQ * max(pitch, SSM_PITCH);              // each of the two areas serves twice
    float* sC = so_sh;
    float* sS = so_sh + area;
    ssm_stage(sC, pitch, base + p.c_col + g * N, p.ld, nt, N, tid, 128);
    const float* pv = p.prev + (((size_t)tile * p.heads + hd) * P + p0) * N;
    for (int i = tid; i < 64 * (N / 4); i += 128) {
        const int r = i / (N / 4), c = (i - r * (N / 4)) * 4;
        gd_copy<16>(sS + ((r & 3) * 16 + (r >> 2)) * pitch + c, pv + (size_t)min(r, wp - 1) * N + c);      // (rows beyond P: never stored)
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float* steps = p.steps + ((size_t)tile * p.heads + hd) * 3 * SSQ;
    if (tid < SSQ) { s_c[tid] = steps[tid]; s_dt[tid] = steps[SSQ + tid]; }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int px = tid & 15, ty = tid >> 4;
    float acc[8][4];
    ssm_dot_tile(sC, sS, pitch, N, ty, px, acc);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const float f = expf(s_c[ty + 8 * i]);
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] *= f;
    }
    __syncthreads();                                           // both areas are free
    float* sM = so_sh;
    float* sX = so_sh + area;
    ssm_stage(sX, SSM_PITCH, base + p.x_col + hd * P + p0, p.ld, nt, wp, tid, 128);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float* sc = p.scores + ((size_t)tile * p.groups + g) * SSQ * SSQ;
    for (int i = tid; i < SSQ * SSQ / 4; i += 128) {           // the weights of the chunk's own tokens
        const int t = i >> 4, s = (i & 15) * 4;
        float4 v = *reinterpret_cast<const float4*>(sc + i * 4);
        const float ct = s_c[t];
        v.x = s <= t ? v.x * s_dt[s] * expf(ct - s_c[s]) : 0.f;
        v.y = s + 1 <= t ? v.y * s_dt[s + 1] * expf(ct - s_c[s + 1]) : 0.f;
        v.z = s + 2 <= t ? v.z * s_dt[s + 2] * expf(ct - s_c[s + 2]) : 0.f;
        v.w = s + 3 <= t ? v.w * s_dt[s + 3] * expf(ct - s_c[s + 3]) : 0.f;
        *reinterpret_cast<float4*>(sM + t * SSM_PITCH + s) = v;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int pc = 4 * px;
    for (int s = 0; s < SSQ; s += 4) {
        float4 x[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) x[k] = *reinterpret_cast<const float4*>(sX + (s + k) * SSM_PITCH + pc);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float4 m = *reinterpret_cast<const float4*>(sM + (ty + 8 * i) * SSM_PITCH + s);
            acc[i][0] = fmaf(m.x, x[0].x, fmaf(m.y, x[1].x, fmaf(m.z, x[2].x, fmaf(m.w, x[3].x, acc[i][0]))));
            acc[i][1] = fmaf(m.x, x[0].y, fmaf(m.y, x[1].y, fmaf(m.z, x[2].y, fmaf(m.w, x[3].y, acc[i][1]))));
            acc[i][2] = fmaf(m.x, x[0].z, fmaf(m.y, x[1].z, fmaf(m.z, x[2].z, fmaf(m.w, x[3].z, acc[i][2]))));
            acc[i][3] = fmaf(m.x, x[0].w, fmaf(m.y, x[1].w, fmaf(m.z, x[2].w, fmaf(m.w, x[3].w, acc[i][3]))));
        }
    }
    if (pc >= wp) return;
    const float d = p.d_skip[hd];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = ty + 8 * i;
        if (t >= nt) continue;
        const float4 x = *reinterpret_cast<const float4*>(sX + t * SSM_PITCH + pc);
        *reinterpret_cast<float4*>(p.out + (size_t)(row0 + t) * p.heads * P + hd * P + p0 + pc) =
            make_float4(fmaf(d, x.x, acc[i][0]), fmaf(d, x.y, acc[i][1]), fmaf(d, x.z, acc[i][2]), fmaf(d, x.w, acc[i][3]));
    }
}

extern "C" int cml_ssm_chunks(const float* rows, long ld, int x_col, int b_col, int c_col, const float* gates, long ldg, const float* a_log,
                              const float* d_skip, const int* tile_seq, const int* tile_q0, int n_tiles, const int* seq_row0,
                              const int* seq_new, const int* seq_start, const int* seq_slot, float* state, float* scores, float* steps,
                              float* prev, float* out, int n_seqs, int heads, int groups, int N, int P, void* stream) {
    if (n_tiles <= 0 || n_seqs <= 0) return 0;
    if (heads < 1 || heads > 65535 || groups < 1 || heads % groups || N < 4 || N > 256 || (N & 3) || P < 4 || (P & 3)) return CML_ERR_BAD_SIZE;
    if (((x_col | b_col | c_col) & 3) || (ld & 3)) return CML_ERR_BAD_ALIGN;
    if ((((uintptr_t)rows) | ((uintptr_t)state) | ((uintptr_t)scores) | ((uintptr_t)steps) | ((uintptr_t)prev) | ((uintptr_t)out)) & 15) return CML_ERR_BAD_ALIGN;
    SsmChunks p = {rows, ld, x_col, b_col, c_col, gates, ldg, a_log, d_skip, tile_seq, tile_q0, seq_row0, seq_new, seq_start, seq_slot,
                   state, scores, steps, prev, out, heads, groups, N, P};
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem_dot = (size_t)2 * SSQ * (N + 4) * sizeof(float);
    const size_t smem_out = (size_t)2 * SSQ * (N + 4 > SSM_PITCH ? N + 4 : SSM_PITCH) * sizeof(float);
    if (smem_dot > 48 * 1024 && cml_allow_smem<ssm_scores_kernel>(smem_dot) != cudaSuccess) return CML_ERR_BAD_SIZE;
    if (smem_out > 48 * 1024 && cml_allow_smem<ssm_outputs_kernel>(smem_out) != cudaSuccess) return CML_ERR_BAD_SIZE;
    constexpr size_t smem_states = (size_t)2 * SSQ * (SST_P + SST_N + 2) * sizeof(float);
    if (cml_allow_smem<ssm_states_kernel>(smem_states) != cudaSuccess) return CML_ERR_BAD_SIZE;
    launch_pdl(ssm_scores_kernel, dim3(n_tiles, groups), dim3(128), smem_dot, s, p);
    launch_pdl(ssm_states_kernel, dim3(n_seqs, heads, ((P + SST_P - 1) / SST_P) * ((N + SST_N - 1) / SST_N)), dim3(128), smem_states, s, p);
    launch_pdl(ssm_outputs_kernel, dim3(n_tiles, heads, (P + 63) / 64), dim3(128), smem_out, s, p);
    return cml_launch_status();
}

// ------------------------------------------------------------------------------------
// The generalized delta rule by chunks of GDC = 16 tokens, for steps that bring several tokens per sequence. With
// W_t the product of the decays of the chunk's tokens up to t (per key channel; W_0 = 1) and S_t = diag(W_t) Z_t the rule is
//
//   Z_t = Z_(t-1) - al_t (be_t^T Z_(t-1)) + ka_t v_t^T,     al = a * u / W_t,  be = u * W_(t-1),  ka = k / W_t,  rh = r * W_t
//
// so with M = be al^T, N = be ka^T (strictly lower triangles), Qa = rh al^T, Qk = rh ka^T (with the diagonal), S the state
// before the chunk and P = be^T Z row by row:
//
//   (I + M) P = be S + N V     =>  P = B' S + N' V,    B' = (I + M)^-1 be,  N' = (I + M)^-1 N
//   O = rh S + Qk V - Qa P     =  R' S + E V,          R' = rh - Qa B',     E = Qk - Qa N'
//   S <- diag(W) (S + ka^T V - al^T P) = diag(W) S + G^T V - A'^T (B' S),   A' = al * W,  G = (ka - N'^T al) * W
//
// Everything but the three products with S and V is made by the first kernel for all chunks side by side; the
// second walks a sequence's chunks with the state in registers. All in float: a decay is at least exp(-rate), so W stays
// above exp(-16 rate), and every al, ka meets the be, rh of a later token, so no product grows.
#define GDC 16
#define GDC_FLOATS(D, Dv) ((size_t)(4 * GDC + 1) * (D) + GDC * GDC + GDC * (Dv))      // B', R', G, A', W, E, V of a (chunk, head)

struct DeltaChunks {
    const float* proj; long ld; int n_splits; long split_stride;
    const float* high; int n_high; long high_stride;
    const float* a_bias; const float* w0;
    float rate;
    const int* tile_seq; const int* tile_q0; const int* seq_row0; const int* seq_new;
    float* chunks; float* gate_out;
    int heads, D, Dv;
};

#define GDP 20               // floats of a row of a 16 x 16 matrix in shared memory (16-byte rows, read four at a time)

// One block per (chunk, head); THREADS >= D, a thread owns a key channel. All of a thread's inputs are asked for before
// any of them is used.
template <int THREADS>
__global__ void __launch_bounds__(THREADS) delta_chunks_kernel(const DeltaChunks p) {
    constexpr int NT = 256 / THREADS;                      // pairs of tokens (t, j) of a thread
    extern __shared__ __align__(16) float dc_sh[];
    __shared__ __align__(16) float sM[GDC][GDP], sN[GDC][GDP], sQk[GDC][GDP], sQa[GDC][GDP], sNt[GDC][GDP];
    __shared__ float s_inv[GDC];
    pdl_wait();
    pdl_launch_dependents();
    const int tile = blockIdx.x, hd = blockIdx.y, D = p.D, Dv = p.Dv, HD = p.heads * D, HV = p.heads * Dv;
    const int seq = p.tile_seq[tile], q0 = p.tile_q0[tile];
    const int nt = min(GDC, p.seq_new[seq] - q0), row0 = p.seq_row0[seq] + q0;
    const int pitch = D + 4, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float* be = dc_sh;
    float* al = be + GDC * pitch;
    float* ka = al + GDC * pitch;
    float* rh = ka + GDC * pitch;
    float* out = p.chunks + ((size_t)tile * p.heads + hd) * GDC_FLOATS(D, Dv);
    const int d = min(tid, D - 1), c = hd * D + d;
    const bool mine = tid < D;
    float kk[GDC], rr[GDC], aa[GDC], zz[GDC];
#pragma unroll
    for (int t = 0; t < GDC; ++t) {
        const float* row = p.proj + (size_t)(row0 + min(t, nt - 1)) * p.ld + c;
        kk[t] = row[HD];
        rr[t] = row[0];
        aa[t] = row[2 * HD + HV];
        zz[t] = p.high[(size_t)(row0 + min(t, nt - 1)) * HD + c];
    }
    for (int sp = 1; sp < p.n_splits; ++sp)                // (products of few rows come as split sums)
#pragma unroll
        for (int t = 0; t < GDC; ++t) {
            const float* row = p.proj + (size_t)sp * p.split_stride + (size_t)(row0 + min(t, nt - 1)) * p.ld + c;
            kk[t] += row[HD];
            rr[t] += row[0];
            aa[t] += row[2 * HD + HV];
        }
    for (int sp = 1; sp < p.n_high; ++sp)
#pragma unroll
        for (int t = 0; t < GDC; ++t) zz[t] += p.high[(size_t)sp * p.high_stride + (size_t)(row0 + min(t, nt - 1)) * HD + c];
    const float ab = p.a_bias[c], w0 = p.w0[c];
    if (mine) {
#pragma unroll
        for (int t = 0; t < GDC; ++t) {
            if (t >= nt) kk[t] = 0.f;
            ka[t * pitch + d] = kk[t];
        }
    }
    for (int e = tid; e < Dv; e += THREADS) {              // the values, and the gate's inputs
        float v[GDC];
        const float* col = p.proj + (size_t)row0 * p.ld + 2 * HD + hd * Dv + e;
#pragma unroll
        for (int t = 0; t < GDC; ++t) v[t] = split_sum(col + (size_t)min(t, nt - 1) * p.ld, p.n_splits, p.split_stride);
#pragma unroll
        for (int t = 0; t < GDC; ++t) out[(4 * GDC + 1) * D + GDC * GDC + t * Dv + e] = t < nt ? v[t] : 0.f;
        if (p.gate_out)
            for (int t = 0; t < nt; ++t)
                p.gate_out[(size_t)(row0 + t) * HV + hd * Dv + e] = split_sum(col + (size_t)t * p.ld + HD + HV, p.n_splits, p.split_stride);
    }
    __syncthreads();
    for (int t = warp; t < GDC; t += THREADS / 32) {
        float ss = 0.f;
        for (int i = lane; i < D; i += 32) ss = fmaf(ka[t * pitch + i], ka[t * pitch + i], ss);
        ss = warp_sum(ss);
        if (lane == 0) s_inv[t] = 1.0f / sqrtf(ss + 1e-6f);
    }
    __syncthreads();
    float W = 1.0f;
    if (mine) {
#pragma unroll
        for (int t = 0; t < GDC; ++t) {
            const bool there = t < nt;                     // tokens that are not there change nothing
            const float w = there ? expf(-p.rate * sigmoid_f(zz[t] + w0)) : 1.0f;
            const float u = kk[t] * s_inv[t];
            be[t * pitch + d] = u * W;
            W *= w;
            const float inv = 1.0f / W;
            al[t * pitch + d] = there ? sigmoid_f(aa[t] + ab) * u * inv : 0.f;
            ka[t * pitch + d] = kk[t] * inv;
            rh[t * pitch + d] = there ? rr[t] * W : 0.f;
        }
        out[4 * GDC * D + d] = W;
    }
    __syncthreads();
    {   // the four products of a pair of tokens (t, j); a thread's pairs share j
        const int j = tid & 15;
        float m[NT], n[NT], qk[NT], qa[NT];
#pragma unroll
        for (int u = 0; u < NT; ++u) m[u] = n[u] = qk[u] = qa[u] = 0.f;
        for (int i = 0; i < D; i += 4) {
            const float4 a = *reinterpret_cast<const float4*>(al + j * pitch + i), k = *reinterpret_cast<const float4*>(ka + j * pitch + i);
#pragma unroll
            for (int u = 0; u < NT; ++u) {
                const int t = (tid >> 4) + u * (THREADS / 16);
                const float4 b = *reinterpret_cast<const float4*>(be + t * pitch + i), r = *reinterpret_cast<const float4*>(rh + t * pitch + i);
                m[u] = fmaf(b.x, a.x, fmaf(b.y, a.y, fmaf(b.z, a.z, fmaf(b.w, a.w, m[u]))));
                n[u] = fmaf(b.x, k.x, fmaf(b.y, k.y, fmaf(b.z, k.z, fmaf(b.w, k.w, n[u]))));
                qk[u] = fmaf(r.x, k.x, fmaf(r.y, k.y, fmaf(r.z, k.z, fmaf(r.w, k.w, qk[u]))));
                qa[u] = fmaf(r.x, a.x, fmaf(r.y, a.y, fmaf(r.z, a.z, fmaf(r.w, a.w, qa[u]))));
            }
        }
#pragma unroll
        for (int u = 0; u < NT; ++u) {
            const int t = (tid >> 4) + u * (THREADS / 16);
            sM[t][j] = j < t ? m[u] : 0.f;
            sN[t][j] = j < t ? n[u] : 0.f;
            sQk[t][j] = j <= t ? qk[u] : 0.f;
            sQa[t][j] = j <= t ? qa[u] : 0.f;
        }
    }
    __syncthreads();
    // x <- (I + M)^-1 x for a column x
    auto solve = [&](float (&x)[GDC]) {
#pragma unroll
        for (int t = 1; t < GDC; ++t)
#pragma unroll
            for (int j = 0; j < t; j += 4) {
                const float4 v = *reinterpret_cast<const float4*>(&sM[t][j]);
                x[t] = fmaf(-v.x, x[j], x[t]);
                if (j + 1 < t) x[t] = fmaf(-v.y, x[j + 1], x[t]);
                if (j + 2 < t) x[t] = fmaf(-v.z, x[j + 2], x[t]);
                if (j + 3 < t) x[t] = fmaf(-v.w, x[j + 3], x[t]);
            }
    };
    float x[GDC];
    if (mine) {                                            // B', then R', column by column
#pragma unroll
        for (int t = 0; t < GDC; ++t) x[t] = be[t * pitch + d];
        solve(x);
#pragma unroll
        for (int t = 0; t < GDC; ++t) {
            float v = rh[t * pitch + d];
#pragma unroll
            for (int j = 0; j <= t; j += 4) {
                const float4 q = *reinterpret_cast<const float4*>(&sQa[t][j]);
                v = fmaf(-q.x, x[j], v);
                if (j + 1 <= t) v = fmaf(-q.y, x[j + 1], v);
                if (j + 2 <= t) v = fmaf(-q.z, x[j + 2], v);
                if (j + 3 <= t) v = fmaf(-q.w, x[j + 3], v);
            }
            out[t * D + d] = x[t];
            out[(GDC + t) * D + d] = v;
        }
    }
    if (tid >= THREADS - 32 && lane < GDC) {               // the last warp: N' column by column, both ways round
#pragma unroll
        for (int t = 0; t < GDC; ++t) x[t] = sN[t][lane];
        solve(x);
        __syncwarp(0xffff);
#pragma unroll
        for (int t = 0; t < GDC; ++t) { sN[t][lane] = x[t]; sNt[lane][t] = x[t]; }
    }
    __syncthreads();
    if (mine) {
#pragma unroll
        for (int t = 0; t < GDC; ++t) x[t] = al[t * pitch + d];
#pragma unroll
        for (int j = 0; j < GDC; ++j) {
            float v = ka[j * pitch + d];
#pragma unroll
            for (int t0 = (j + 1) & ~3; t0 < GDC; t0 += 4) {
                const float4 q = *reinterpret_cast<const float4*>(&sNt[j][t0]);
                if (t0 > j) v = fmaf(-q.x, x[t0], v);
                if (t0 + 1 > j) v = fmaf(-q.y, x[t0 + 1], v);
                if (t0 + 2 > j) v = fmaf(-q.z, x[t0 + 2], v);
                if (t0 + 3 > j) v = fmaf(-q.w, x[t0 + 3], v);
            }
            out[(2 * GDC + j) * D + d] = v * W;
            out[(3 * GDC + j) * D + d] = x[j] * W;
        }
    }
    for (int i = tid; i < GDC * GDC; i += THREADS) {
        const int t = i >> 4, j = i & 15;
        float v = sQk[t][j];
        for (int q = j + 1; q <= t; ++q) v = fmaf(-sQa[t][q], sN[q][j], v);
        out[(4 * GDC + 1) * D + i] = v;
    }
}

extern "C" int cml_delta_chunks(const float* proj, long ld, int n_splits, long split_stride, const float* high, int n_high,
                                long high_stride, const float* a_bias, const float* w0, float rate, const int* tile_seq,
                                const int* tile_q0, int n_tiles, const int* seq_row0, const int* seq_new, float* chunks,
                                float* gate_out, int heads, int D, int Dv, void* stream) {
    if (n_tiles <= 0) return 0;
    if (heads < 1 || heads > 65535 || D < 4 || D > 256 || (D & 3) || Dv < 4 || (Dv & 3) || n_splits < 1 || n_high < 1 || rate < 0.f || rate > 2.f)
        return CML_ERR_BAD_SIZE;
    DeltaChunks p = {proj, ld, n_splits, split_stride, high, n_high, high_stride, a_bias, w0, rate, tile_seq, tile_q0, seq_row0, seq_new,
                     chunks, gate_out, heads, D, Dv};
    const size_t smem = (size_t)4 * GDC * (D + 4) * sizeof(float);
    if (D <= 128) {
        launch_pdl(delta_chunks_kernel<128>, dim3(n_tiles, heads), dim3(128), smem, (cudaStream_t)stream, p);
    } else {
        if (smem > 32 * 1024 && cml_allow_smem<delta_chunks_kernel<256>>(smem) != cudaSuccess) return CML_ERR_BAD_SIZE;
        launch_pdl(delta_chunks_kernel<256>, dim3(n_tiles, heads), dim3(256), smem, (cudaStream_t)stream, p);
    }
    return cml_launch_status();
}

// The walk over a sequence's chunks. A warp owns COLS columns of the state of one (sequence, head): NS lanes of DS key
// channels each hold CPT columns, and 32 / NS such groups stand side by side. The products with the state give every lane
// partial sums over its channels for 32 / CPT rows at a time; they are added over the lanes by halving (each step
// hands half of the values over, so a lane ends with sums of its own), in a fixed order. The chunk's matrices come by
// cp.async into one of two buffers while the other one's chunk is worked on.
struct ChunkScan {
    const float* chunks; float* state;
    const int* seq_new; const int* seq_row0; const int* seq_start; const int* seq_slot;
    float* out;
    int heads, D, Dv;
};

template <int DS, int NS, int CPT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) delta_chunk_scan_kernel(const ChunkScan p) {
    constexpr int G = 32 / NS, WCOLS = G * CPT, COLS = WARPS * WCOLS;
    constexpr int RG = NS / CPT;                           // rows of a group: its RG x CPT sums end in its NS lanes
    constexpr int DP = NS * DS;
    constexpr int THREADS = WARPS * 32;
    extern __shared__ __align__(16) float cs_sh[];
    const int D = p.D, Dv = p.Dv, heads = p.heads;
    constexpr int BUF = (4 * GDC + 1) * DP + GDC * GDC + GDC * COLS;
    float* sP = cs_sh + 2 * BUF;                           // [GDC][COLS]: B' S
    pdl_wait();
    pdl_launch_dependents();
    const int s = blockIdx.x, hd = blockIdx.y, col0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int group = lane / NS, slice = lane % NS, d0 = slice * DS;
    const int n = p.seq_new[s], row0 = p.seq_row0[s];
    const bool fresh = p.seq_start[s] == 0;
    int first = 0;                                         // chunks of the sequences before this one
    for (int q = 0; q < s; ++q) first += (p.seq_new[q] + GDC - 1) / GDC;
    const int n_chunks = (n + GDC - 1) / GDC;
    const int wc = warp * WCOLS + group * CPT;             // this lane's first column within the block
    float S[CPT][DS];
    size_t cell[CPT];
    bool live[CPT];
#pragma unroll
    for (int e = 0; e < CPT; ++e) {
        live[e] = col0 + wc + e < Dv && d0 < D;
        cell[e] = (((size_t)p.seq_slot[s] * heads + hd) * Dv + (col0 + wc + e < Dv ? col0 + wc + e : 0)) * D + (d0 < D ? d0 : 0);
#pragma unroll
        for (int i = 0; i < DS; i += 4) {
            const bool ok = live[e] && d0 + i < D && !fresh;
            const float4 t = *reinterpret_cast<const float4*>(p.state + cell[e] + (ok ? i : 0));
            S[e][i] = ok ? t.x : 0.f; S[e][i + 1] = ok ? t.y : 0.f; S[e][i + 2] = ok ? t.z : 0.f; S[e][i + 3] = ok ? t.w : 0.f;
        }
    }
    if (D < DP || Dv - col0 < COLS) {                      // channels and columns that are not there stay zero
        for (int i = tid; i < 2 * BUF; i += THREADS) cs_sh[i] = 0.f;
        __syncthreads();
    }
    auto fetch = [&](int ch, int buf) {
        const float* src = p.chunks + ((size_t)(first + ch) * heads + hd) * GDC_FLOATS(D, Dv);
        float* dst = cs_sh + buf * BUF;
        if (D == DP) {                                     // all matrices and E in one run of memory
            for (int i = tid * 4; i < (4 * GDC + 1) * DP + GDC * GDC; i += THREADS * 4) gd_copy<16>(dst + i, src + i);
        } else {
            for (int r = warp; r < 4 * GDC + 1; r += WARPS)
                for (int i = lane * 4; i < D; i += 128) gd_copy<16>(dst + r * DP + i, src + (size_t)r * D + i);
            for (int i = tid * 4; i < GDC * GDC; i += THREADS * 4) gd_copy<16>(dst + (4 * GDC + 1) * DP + i, src + (size_t)(4 * GDC + 1) * D + i);
        }
        const float* v = src + (size_t)(4 * GDC + 1) * D + GDC * GDC + col0;
        for (int i = tid; i < GDC * COLS / 4; i += THREADS) {
            const int t = i / (COLS / 4), e = (i % (COLS / 4)) * 4;
            if (col0 + e < Dv) gd_copy<16>(dst + (4 * GDC + 1) * DP + GDC * GDC + t * COLS + e, v + (size_t)t * Dv + e);
        }
    };
    fetch(0, 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int ch = 0; ch < n_chunks; ++ch) {
        if (ch + 1 < n_chunks) fetch(ch + 1, (ch + 1) & 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");       // all but the newest group: this chunk is here
        __syncthreads();
        const float* m = cs_sh + (ch & 1) * BUF;
        const float* sE = m + (4 * GDC + 1) * DP;
        const float* sV = sE + GDC * GDC;
        const int nt = min(GDC, n - ch * GDC);
        // B' S and R' S, RG rows at a time
#pragma unroll
        for (int rg = 0; rg < 2 * GDC; rg += RG) {
            float acc[NS];                                 // value r * CPT + e: row rg + r, column e
#pragma unroll
            for (int r = 0; r < RG; ++r) {
#pragma unroll
                for (int e = 0; e < CPT; ++e) acc[r * CPT + e] = 0.f;
#pragma unroll
                for (int i = 0; i < DS; i += 4) {
                    const float4 b = *reinterpret_cast<const float4*>(m + (rg + r) * DP + d0 + i);
#pragma unroll
                    for (int e = 0; e < CPT; ++e)
                        acc[r * CPT + e] = fmaf(b.x, S[e][i], fmaf(b.y, S[e][i + 1], fmaf(b.z, S[e][i + 2], fmaf(b.w, S[e][i + 3], acc[r * CPT + e]))));
                }
            }
#pragma unroll
            for (int h = NS / 2; h > 0; h >>= 1) {         // lane bit h keeps the upper half of what is left
                const bool up = (slice & h) != 0;
#pragma unroll
                for (int i = 0; i < h; ++i) {
                    const float give = up ? acc[i] : acc[i + h], keep = up ? acc[i + h] : acc[i];
                    acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, h);
                }
            }
            const int row = rg + slice / CPT, e = slice % CPT;     // the sum this lane ended with
            if (row < GDC) {
                sP[row * COLS + wc + e] = acc[0];
            } else {
                const int t = row - GDC;
                float o = acc[0];
#pragma unroll
                for (int j = 0; j < GDC; j += 4) {
                    const float4 w = *reinterpret_cast<const float4*>(sE + t * GDC + j);
                    o = fmaf(w.x, sV[j * COLS + wc + e], o);
                    o = fmaf(w.y, sV[(j + 1) * COLS + wc + e], o);
                    o = fmaf(w.z, sV[(j + 2) * COLS + wc + e], o);
                    o = fmaf(w.w, sV[(j + 3) * COLS + wc + e], o);
                }
                if (t < nt && col0 + wc + e < Dv)
                    asm volatile("st.global.f32 [%0], %1;" ::"l"(p.out + ((size_t)(row0 + ch * GDC + t) * heads + hd) * Dv + col0 + wc + e), "f"(o));
            }
        }
        __syncwarp();                                      // a warp reads back its own columns of sP
        // S <- diag(W) S + G^T V - A'^T (B' S)
#pragma unroll
        for (int i = 0; i < DS; i += 4) {
            const float4 w = *reinterpret_cast<const float4*>(m + 4 * GDC * DP + d0 + i);
#pragma unroll
            for (int e = 0; e < CPT; ++e) { S[e][i] *= w.x; S[e][i + 1] *= w.y; S[e][i + 2] *= w.z; S[e][i + 3] *= w.w; }
        }
#pragma unroll
        for (int j = 0; j < GDC; ++j) {
            float v[CPT], q[CPT];
            if constexpr (CPT == 4) {                      // (wc is a multiple of 4)
                const float4 vv = *reinterpret_cast<const float4*>(sV + j * COLS + wc), qq = *reinterpret_cast<const float4*>(sP + j * COLS + wc);
                v[0] = vv.x; v[1] = vv.y; v[2] = vv.z; v[3] = vv.w;
                q[0] = -qq.x; q[1] = -qq.y; q[2] = -qq.z; q[3] = -qq.w;
            } else {
#pragma unroll
                for (int e = 0; e < CPT; ++e) { v[e] = sV[j * COLS + wc + e]; q[e] = -sP[j * COLS + wc + e]; }
            }
#pragma unroll
            for (int i = 0; i < DS; i += 4) {
                const float4 g = *reinterpret_cast<const float4*>(m + (2 * GDC + j) * DP + d0 + i), a = *reinterpret_cast<const float4*>(m + (3 * GDC + j) * DP + d0 + i);
#pragma unroll
                for (int e = 0; e < CPT; ++e) {
                    S[e][i] = fmaf(g.x, v[e], fmaf(a.x, q[e], S[e][i]));
                    S[e][i + 1] = fmaf(g.y, v[e], fmaf(a.y, q[e], S[e][i + 1]));
                    S[e][i + 2] = fmaf(g.z, v[e], fmaf(a.z, q[e], S[e][i + 2]));
                    S[e][i + 3] = fmaf(g.w, v[e], fmaf(a.w, q[e], S[e][i + 3]));
                }
            }
        }
        __syncthreads();                                   // before the next fetch overwrites this buffer
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int e = 0; e < CPT; ++e)
#pragma unroll
        for (int i = 0; i < DS; i += 4)
            if (live[e] && d0 + i < D)
                *reinterpret_cast<float4*>(p.state + cell[e] + i) = make_float4(S[e][i], S[e][i + 1], S[e][i + 2], S[e][i + 3]);
}

extern "C" int cml_delta_chunk_scan(const float* chunks, float* state, const int* seq_row0, const int* seq_new, const int* seq_start,
                                    const int* seq_slot, float* out, int n_seqs, int heads, int D, int Dv, void* stream) {
    if (n_seqs <= 0) return 0;
    if (heads < 1 || heads > 65535 || D < 4 || D > 256 || (D & 3) || Dv < 4 || (Dv & 3)) return CML_ERR_BAD_SIZE;
    if ((((uintptr_t)chunks) | ((uintptr_t)state)) & 15) return CML_ERR_BAD_ALIGN;
    ChunkScan p = {chunks, state, seq_new, seq_row0, seq_start, seq_slot, out, heads, D, Dv};
#define CS_CASE(DS_, NS_, CPT_, WARPS_)                                                                                            \
    if (D <= NS_ * DS_) {                                                                                                          \
        constexpr int COLS = WARPS_ * (32 / NS_) * CPT_;                                                                           \
        constexpr size_t smem = (size_t)(2 * ((4 * GDC + 1) * NS_ * DS_ + GDC * GDC + GDC * COLS) + GDC * COLS) * sizeof(float);   \
        if (smem > 48 * 1024 && cml_allow_smem<delta_chunk_scan_kernel<DS_, NS_, CPT_, WARPS_>>(smem) != cudaSuccess) return CML_ERR_BAD_SIZE; \
        launch_pdl(delta_chunk_scan_kernel<DS_, NS_, CPT_, WARPS_>, dim3(n_seqs, heads, (Dv + COLS - 1) / COLS), dim3(WARPS_ * 32), smem, \
                   (cudaStream_t)stream, p);                                                                                       \
        return cml_launch_status();                                                                                                \
    }
    CS_CASE(4, 8, 2, 2) CS_CASE(4, 16, 2, 4) CS_CASE(4, 32, 4, 4) CS_CASE(8, 32, 4, 4)
#undef CS_CASE
    return CML_ERR_BAD_SIZE;
}

// ------------------------------------------------------------------------------------
// Rotation of heads inside float rows, in place: x [rows, ld] holds `heads` heads of D channels from column col0; the
// first rot_dim channels of every head are turned by angle = position * inv_freq[i] (pairing 1: channels (2i, 2i + 1);
// 0: channels (i, i + rot_dim / 2)), sines and cosines times `amp`; then heads from number `scaled_from` on are
// multiplied by `scale` (all their channels). A warp owns one (row, head); both members of a pair are read before
// either is written.
__global__ void rotate_rows_kernel(float* __restrict__ x, long ld, int col0, int rows, int heads, int D, int rot_dim,
                                   int pairing, const float* __restrict__ inv_freq, float amp, const int* __restrict__ row_pos,
                                   int scaled_from, float scale) {
    pdl_wait();
    pdl_launch_dependents();
    const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    if (warp >= rows * heads) return;
    const int r = warp / heads, hd = warp % heads;
    float* h = x + (size_t)r * ld + col0 + (size_t)hd * D;
    const float pos = (float)row_pos[r];
    const float mul = hd >= scaled_from ? scale : 1.0f;
    const int half = rot_dim / 2;
    for (int i = lane; i < half; i += 32) {
        const int a = pairing ? 2 * i : i, b = pairing ? 2 * i + 1 : i + half;
        float sn, cs;
        sincosf(pos * inv_freq[i], &sn, &cs);
        sn *= amp; cs *= amp;
        const float u = h[a], v = h[b];
        h[a] = (u * cs - v * sn) * mul;
        h[b] = (v * cs + u * sn) * mul;
    }
    if (mul != 1.0f)
        for (int c = rot_dim + lane; c < D; c += 32) h[c] *= mul;
}

extern "C" int cml_rotate_rows(float* x, long ld, int col0, int rows, int heads, int D, int rot_dim, int pairing,
                               const float* inv_freq, float amp, const int* row_pos, int scaled_from, float scale, void* stream) {
    if (rows <= 0 || heads <= 0) return 0;
    if (rot_dim < 0 || rot_dim > D || (rot_dim & 1)) return CML_ERR_BAD_SIZE;
    const long warps = (long)rows * heads;
    launch_pdl(rotate_rows_kernel, dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, (cudaStream_t)stream, x, ld, col0, rows, heads,
               D, rot_dim, pairing, inv_freq, amp, row_pos, scaled_from, scale);
    return cml_launch_status();
}

// ------------------------------------------------------------------------------------
// After a scan: per (row, head) o = raw / den (den = max(|n . q|, exp(-m)) + 1e-6 where the
// raw rows carry them, else 1), y = o / sqrt(mean(o^2) + eps) * w * sigmoid(gate) (or * silu(gate)), written in
// the compute type for the output projection. A warp owns one (row, head). raw [rows, heads, ldh]
// with ldh = Dv (+ 2 with a denominator); w [Dv] shared by the heads (w_head_stride 0) or
// [heads x Dv]; gate [rows, ldg] at column gate_col + head * Dv.
template <typename TO>
__global__ void head_norm_gate_kernel(const float* __restrict__ raw, int ldh, int with_den, const float* __restrict__ w,
                                      int w_head_stride, const float* __restrict__ gate, long ldg, int gate_col,
                                      TO* __restrict__ out, long ldo, int rows, int heads, int Dv, float eps, int gate_silu) {
    pdl_wait();
    pdl_launch_dependents();
    const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    if (warp >= rows * heads) return;
    const int r = warp / heads, hd = warp % heads;
    const float* x = raw + ((size_t)r * heads + hd) * ldh;
    float inv = 1.0f;
    if (with_den) inv = 1.0f / (fmaxf(fabsf(x[Dv]), expf(-x[Dv + 1])) + 1e-6f);
    float ss = 0.f;
    for (int c = lane; c < Dv; c += 32) {
        const float o = x[c] * inv;
        ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    const float scale = inv / sqrtf(ss / (float)Dv + eps);
    const float* wv = w ? w + (size_t)hd * w_head_stride : nullptr;      // null: a norm without weight
    const float* gt = gate + (size_t)r * ldg + gate_col + hd * Dv;
    TO* o = out + (size_t)r * ldo + (size_t)hd * Dv;
    for (int c = lane; c < Dv; c += 32) o[c] = from_f32<TO>(x[c] * scale * (wv ? wv[c] : 1.0f) * (gate_silu ? silu_f(gt[c]) : sigmoid_f(gt[c])));
}

extern "C" int cml_head_norm_gate(const float* raw, int ldh, int with_den, const float* w, int w_head_stride, const float* gate,
                                  long ldg, int gate_col, void* out, long ldo, int out_dtype, int rows, int heads, int Dv, float eps,
                                  int gate_silu, void* stream) {
    if (rows <= 0) return 0;
    const long warps = (long)rows * heads;
    dim3 grid((unsigned)((warps + 3) / 4));
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == CML_DTYPE_F32)
        launch_pdl(head_norm_gate_kernel<float>, grid, dim3(128), 0, s, raw, ldh, with_den, w, w_head_stride, gate, ldg, gate_col,
                   (float*)out, ldo, rows, heads, Dv, eps, gate_silu);
    else if (out_dtype == CML_DTYPE_BF16)
        launch_pdl(head_norm_gate_kernel<bf16>, grid, dim3(128), 0, s, raw, ldh, with_den, w, w_head_stride, gate, ldg, gate_col,
                   (bf16*)out, ldo, rows, heads, Dv, eps, gate_silu);
    else
        return CML_ERR_BAD_DTYPE;
    return cml_launch_status();
}
