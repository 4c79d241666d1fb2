// linear_recurrence.cu -- sequence mixers whose memory is a fixed-size f32 state per sequence, for ragged steps (portions of prompts
// beside single decoded tokens in one launch).  Entry b's rows continue the sequence whose state sits in slot seq_slots[b];
// seq_start[b] == 0 means "new sequence": what the slot holds is ignored (taken as zero), so a slot is never cleared.
//
//   causal_conv_ex        y[t, c] = act(sum_j taps[c, j] * in[t - K + 1 + j, c] + out_bias[c]) (+ in[t, c]), in = x + in_bias, zeros before
//                         the sequence's start; the K - 1 inputs before a portion come from conv_state [slots, K-1, C], which is then
//                         rolled forward over the portion.  act = none or SiLU; the "+ in" form is a convolution added to its own input.
//   block_diag_linear     out[t, b M + j] = sum_i w[b, j, i] x[t, b N + i] + bias[b M + j]: one matrix per block of N neighbouring
//                         channels, true 32-bit products (the gates of a recurrence).
//   gated_linear_scan     per channel  S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,  a_t = exp(-c r_t softplus(lam)),  r, i = sigmoid of
//                         the block-diagonal products;  out_t = S_t * gelu_tanh(y_t + y_bias).  One kernel for steps of few rows per entry;
//                         for portions of prompts a row-parallel pass first turns gates and y into a_t, the input term and the GELU (in place);
//                         from 512 rows per entry the bare scan that follows runs over chunks of 128 rows, all chunks at once.
//   linear_attention      per head, S [dk, dv]:  S_t = a_t S_(t-1) + b_t k_t v_t^T,  o_t = S_t^T q_t, in two gatings (a third below):
//                           fixed decay      a = decay[h], b = 1;
//                           exponential      a_t = e^(f_t + m_(t-1) - m_t), b_t = e^(i_t - m_t) with the running maximum m_t = max(f_t + m_(t-1), i_t),
//                                            m_0 = 0, i = cap tanh(. / cap), f = logsigmoid(cap tanh(. / cap)); a normaliser n_t = a_t n_(t-1) + b_t k_t
//                                            rides along and o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6).  n and m are stored once per
//                                            block of 16 value columns, so that no block reads what another one writes.
//   linear_attention_channel  the same with a decay per token AND key row, S_t = diag(a_t) S_(t-1) + k_t v_t^T (a handed in as f32 [T, H dk]).
//                         The _bonus form reads a token's output before its decay and write: o_t = (S_(t-1) + diag(bonus) k_t v_t^T)^T q_t.
//   low_rank_map          a second low-rank factor in 32 bits, z = w y + bias (y through tanh or not), as one of: sigmoid(z)^(1/tau), exp(-exp(z)),
//                         exp(-exp(log_rate) softplus(z)), z.  low_rank_decay is the first of them.
//   token_shift_mix       several copies of a row, each moved its own way towards the previous token's row (which is part of the state).
//                         A block of four warps owns 16 value columns of one head of one entry; inside a warp the key rows are split eight
//                         ways (lane = 4 * part + column) with the lane's rows of S (and of n) in registers; tokens come in tiles of 16
//                         staged through shared memory with the activation already applied, the per-token coefficients worked out once
//                         per tile (the chain of maxima by one lane, the exponentials by sixteen).  Every sum has a fixed order, so
//                         portions of any size leave the same state bit for bit.  State S is stored [slot, head, column, row].
#include "common.cuh"

namespace b200 {
namespace {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
    const float c = 0.7978845608028654f;       // sqrt(2 / pi)
    return 0.5f * z * (1.0f + tanhf(c * (z + 0.044715f * z * z * z)));
}

template <typename TOut>
__global__ void __launch_bounds__(128)
causal_conv_ex_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ in_bias, const float* __restrict__ taps,
                      const float* __restrict__ out_bias, const float* __restrict__ conv_state, TOut* __restrict__ y, int64_t ldy,
                      const int32_t* __restrict__ token_seq, const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ seq_slots,
                      const int32_t* __restrict__ seq_start, int C, int K, int act, int add_input) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 128 + threadIdx.x;
    const int t = blockIdx.y;
    if (c >= C) return;
    const int b = token_seq[t];
    const int i = t - cu_seqlens[b];
    const bool fresh = seq_start[b] == 0;
    const float* st = conv_state + (int64_t)seq_slots[b] * (K > 1 ? K - 1 : 1) * C;
    const float ib = in_bias ? in_bias[c] : 0.f;
    float acc = 0.f, cur = 0.f;
    for (int d = K - 1; d >= 0; --d) {            // oldest input first
        const int src = i - d;
        float v;
        if (src >= 0) v = x[(int64_t)(t - d) * ldx + c] + ib;
        else v = fresh ? 0.f : st[(int64_t)(K - 1 + src) * C + c];
        if (d == 0) cur = v;
        acc = fmaf(taps[(int64_t)c * K + (K - 1 - d)], v, acc);
    }
    if (out_bias) acc += out_bias[c];
    if (act == 1) acc = silu_f(acc);
    if (add_input) acc += cur;
    y[(int64_t)t * ldy + c] = from_f32<TOut>(acc);
}

__global__ void __launch_bounds__(128)
causal_conv_roll_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ in_bias, float* __restrict__ conv_state,
                        const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ seq_slots, const int32_t* __restrict__ seq_start, int C, int K) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 128 + threadIdx.x;
    const int b = blockIdx.y;
    if (c >= C) return;
    const int t0 = cu_seqlens[b], n = cu_seqlens[b + 1] - t0;
    if (n <= 0) return;
    const bool fresh = seq_start[b] == 0;
    const float ib = in_bias ? in_bias[c] : 0.f;
    float* st = conv_state + (int64_t)seq_slots[b] * (K - 1) * C;
    // the sequence's inputs so far are [old state rows 0 .. K-2][portion rows 0 .. n-1]; the last K-1 of them stay.  Row j of the new
    // state is element n + j of that list: j ascends and n >= 1, so an old row is read before it is overwritten.
    for (int j = 0; j < K - 1; ++j) {
        const int e = n + j;
        float v;
        if (e >= K - 1) v = x[(int64_t)(t0 + e - (K - 1)) * ldx + c] + ib;
        else v = fresh ? 0.f : st[(int64_t)e * C + c];
        st[(int64_t)j * C + c] = v;
    }
}

// Steps of many rows: a thread walks 16 rows of kV channels with the taps and the inputs of the last kK - 1 rows in registers, so that every input is read once.
// kK is the number of taps rounded up; the taps that do not exist are zero and oldest, so the sum is the one above term by term.
constexpr int kConvRows = 16;
template <typename TOut, int kK, int kV>
__global__ void __launch_bounds__(128)
causal_conv_walk_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ in_bias, const float* __restrict__ taps,
                        const float* __restrict__ out_bias, const float* __restrict__ conv_state, TOut* __restrict__ y, int64_t ldy,
                        const int32_t* __restrict__ token_seq, const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ seq_slots,
                        const int32_t* __restrict__ seq_start, int T, int C, int K, int act, int add_input) {
    pdl_wait();
    pdl_trigger();
    const int c = (blockIdx.x * 128 + threadIdx.x) * kV;
    const int t_begin = blockIdx.y * kConvRows, t_end = min(T, t_begin + kConvRows);
    if (c >= C) return;
    auto load = [&](const float* p, float (&v)[kV]) {
        if constexpr (kV == 4) { const float4 f = *reinterpret_cast<const float4*>(p); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
        else v[0] = *p;
    };
    float w[kK][kV], h[kK][kV], ib[kV], ob[kV];      // taps and inputs, oldest first; h[kK - 1] is the current row
#pragma unroll
    for (int j = 0; j < kV; ++j) {
        ib[j] = in_bias ? in_bias[c + j] : 0.f;
        ob[j] = out_bias ? out_bias[c + j] : 0.f;
#pragma unroll
        for (int k = 0; k < kK; ++k) { const int d = kK - 1 - k; w[k][j] = d < K ? taps[(int64_t)(c + j) * K + (K - 1 - d)] : 0.f; h[k][j] = 0.f; }
    }
    int entry = -1;
    for (int t = t_begin; t < t_end; ++t) {
        const int b = token_seq[t];
        if (b != entry) {                            // the rows before this one: earlier rows of the entry, the state, or nothing
            entry = b;
            const int i = t - cu_seqlens[b];
            const bool fresh = seq_start[b] == 0;
            const float* st = conv_state + (int64_t)seq_slots[b] * (K > 1 ? K - 1 : 1) * C + c;
#pragma unroll
            for (int k = 1; k < kK; ++k) {           // shifted down by one below: h[k] is the row kK - k rows back
                const int src = i - (kK - k);
                if (kK - k >= K || (src < 0 && fresh)) {
#pragma unroll
                    for (int j = 0; j < kV; ++j) h[k][j] = 0.f;
                } else if (src >= 0) {
                    load(x + (int64_t)(t - (kK - k)) * ldx + c, h[k]);
#pragma unroll
                    for (int j = 0; j < kV; ++j) h[k][j] += ib[j];
                } else {
                    load(st + (int64_t)(K - 1 + src) * C, h[k]);
                }
            }
        }
#pragma unroll
        for (int k = 0; k + 1 < kK; ++k)
#pragma unroll
            for (int j = 0; j < kV; ++j) h[k][j] = h[k + 1][j];
        load(x + (int64_t)t * ldx + c, h[kK - 1]);
        float o[kV];
        TOut q[kV];
#pragma unroll
        for (int j = 0; j < kV; ++j) {
            h[kK - 1][j] += ib[j];
            o[j] = 0.f;
#pragma unroll
            for (int k = 0; k < kK; ++k) o[j] = fmaf(w[k][j], h[k][j], o[j]);
            o[j] += ob[j];
            if (act == 1) o[j] = silu_f(o[j]);
            if (add_input) o[j] += h[kK - 1][j];
            q[j] = from_f32<TOut>(o[j]);
        }
        TOut* dst = y + (int64_t)t * ldy + c;
        if constexpr (kV == 1) *dst = q[0];
        else if constexpr (sizeof(TOut) == 4) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(q);
        else *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(q);
    }
}

// Steps in which every entry brings one row: the convolution and the roll of the state in one kernel (a thread owns its channel's state column)
template <typename TOut>
__global__ void __launch_bounds__(128)
causal_conv_step_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ in_bias, const float* __restrict__ taps,
                        const float* __restrict__ out_bias, float* __restrict__ conv_state, TOut* __restrict__ y, int64_t ldy,
                        const int32_t* __restrict__ seq_slots, const int32_t* __restrict__ seq_start, int C, int K, int act, int add_input) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 128 + threadIdx.x;
    const int b = blockIdx.y;
    if (c >= C) return;
    const bool fresh = seq_start[b] == 0;
    float* st = conv_state + (int64_t)seq_slots[b] * (K > 1 ? K - 1 : 1) * C;
    const float cur = x[(int64_t)b * ldx + c] + (in_bias ? in_bias[c] : 0.f);
    float acc = 0.f;
    for (int j = 0; j < K - 1; ++j) {             // oldest input first; row j moves to row j - 1
        const float v = fresh ? 0.f : st[(int64_t)j * C + c];
        acc = fmaf(taps[(int64_t)c * K + j], v, acc);
        if (j > 0) st[(int64_t)(j - 1) * C + c] = v;
    }
    if (K > 1) st[(int64_t)(K - 2) * C + c] = cur;
    acc = fmaf(taps[(int64_t)c * K + K - 1], cur, acc);
    if (out_bias) acc += out_bias[c];
    if (act == 1) acc = silu_f(acc);
    if (add_input) acc += cur;
    y[(int64_t)b * ldy + c] = from_f32<TOut>(acc);
}

// ---- block-diagonal f32 product ---------------------------------------------------------------------------------------------------
constexpr int kBM = 64, kBN = 64, kBK = 16;

__global__ void __launch_bounds__(256)
block_diag_linear_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ y,
                         int64_t ldy, int T, int M, int N) {
    pdl_wait();
    pdl_trigger();
    __shared__ float xs[kBK][kBM + 4], ws[kBK][kBN + 4];
    const int blk = blockIdx.z;
    const float* xb = x + (int64_t)blk * N;
    const float* wb = w + (int64_t)blk * M * N;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int row0 = blockIdx.y * kBM, col0 = blockIdx.x * kBN;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < N; k0 += kBK) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int idx = threadIdx.x + i * 256, r = idx >> 4, c = idx & 15;
            const int gr = row0 + r, gc = k0 + c, wr = col0 + r;
            xs[c][r] = (gr < T && gc < N) ? xb[(int64_t)gr * ldx + gc] : 0.f;
            ws[c][r] = (wr < M && gc < N) ? wb[(int64_t)wr * N + gc] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < kBK; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xs[kk][ty * 4 + i]; b[i] = ws[kk][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int gr = row0 + ty * 4 + i;
        if (gr >= T) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int gc = col0 + tx * 4 + j;
            if (gc < M) y[(int64_t)gr * ldy + (int64_t)blk * M + gc] = acc[i][j] + (bias ? bias[(int64_t)blk * M + gc] : 0.f);
        }
    }
}

// few rows: a warp owns one output column of one block and up to 4 rows, lanes stride the block's inputs
__global__ void __launch_bounds__(256)
block_diag_rows_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ y,
                       int64_t ldy, int T, int M, int N) {
    pdl_wait();
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int blk = blockIdx.z;
    const int col = blockIdx.x * 8 + warp;
    const int r0 = blockIdx.y * 4;
    if (col >= M) return;
    const float* wr = w + ((int64_t)blk * M + col) * N;
    const float* xb = x + (int64_t)blk * N;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int i = lane; i < N; i += 32) {
        const float wv = wr[i];
#pragma unroll
        for (int r = 0; r < 4; ++r)
            if (r0 + r < T) acc[r] = fmaf(xb[(int64_t)(r0 + r) * ldx + i], wv, acc[r]);
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const float s = warp_sum(acc[r]);
        if (lane == 0 && r0 + r < T) y[(int64_t)(r0 + r) * ldy + (int64_t)blk * M + col] = s + (bias ? bias[(int64_t)blk * M + col] : 0.f);
    }
}

// ---- the gated scan ------------------------------------------------------------------------------------------------------------------
// One thread per (entry, channel); the next rows' operands are fetched while the current row is applied.  gates f32 [T, blocks, 2 n]: per
// block the recurrence gate's pre-activations, then the input gate's.
template <typename TOut>
__global__ void __launch_bounds__(64)
gated_linear_scan_kernel(const float* __restrict__ u, int64_t ldu, const float* __restrict__ gates, int64_t ldg, const float* __restrict__ lam,
                         const float* __restrict__ ypre, int64_t ldy, const float* __restrict__ y_bias, float* __restrict__ state, TOut* __restrict__ out,
                         const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ seq_slots, const int32_t* __restrict__ seq_start, int C, int n,
                         float decay_scale) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 64 + threadIdx.x;
    const int b = blockIdx.y;
    if (c >= C) return;
    const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
    if (t1 <= t0) return;
    float* sp = state + (int64_t)seq_slots[b] * C + c;
    float S = seq_start[b] == 0 ? 0.f : *sp;
    const float k = -decay_scale * softplus_f(lam[c]);
    const float yb = y_bias ? y_bias[c] : 0.f;
    const int blk = c / n, j = c - blk * n;
    const int rc = blk * 2 * n + j, ic = rc + n;
    constexpr int kAhead = 4;
    float gr[kAhead], gi[kAhead], uu[kAhead], yy[kAhead];
#pragma unroll
    for (int a = 0; a < kAhead; ++a) {
        const int t = min(t0 + a, t1 - 1);
        gr[a] = gates[(int64_t)t * ldg + rc]; gi[a] = gates[(int64_t)t * ldg + ic]; uu[a] = u[(int64_t)t * ldu + c]; yy[a] = ypre[(int64_t)t * ldy + c];
    }
    for (int tb = t0; tb < t1; tb += kAhead) {
        float cr[kAhead], ci[kAhead], cu[kAhead], cy[kAhead];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) { cr[a] = gr[a]; ci[a] = gi[a]; cu[a] = uu[a]; cy[a] = yy[a]; }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int t = min(tb + kAhead + a, t1 - 1);
            gr[a] = gates[(int64_t)t * ldg + rc]; gi[a] = gates[(int64_t)t * ldg + ic]; uu[a] = u[(int64_t)t * ldu + c]; yy[a] = ypre[(int64_t)t * ldy + c];
        }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            if (tb + a >= t1) break;
            const float la = k * sigmoid_f(cr[a]);                     // log a_t <= 0
            const float at = expf(la);
            const float mult = sqrtf(-expm1f(2.0f * la));               // sqrt(1 - a^2) without cancellation near a = 1
            S = fmaf(at, S, mult * sigmoid_f(ci[a]) * cu[a]);
            out[(int64_t)(tb + a) * C + c] = from_f32<TOut>(S * gelu_tanh_f(cy[a] + yb));
        }
    }
    *sp = S;
}

// Portions of prompts: the per-token part (two sigmoids, the decay and its square-root complement, the GELU of the other branch) is done for all
// rows at once, in place -- gates[t, blk, j] <- a_t, gates[t, blk, n + j] <- sqrt(1 - a_t^2) i_t u_t, y[t, c] <- gelu_tanh(y + bias) -- and the scan
// itself is two multiply-adds per row with the next rows' operands in flight.
__global__ void gated_scan_prepare_kernel(const float* __restrict__ u, int64_t ldu, float* __restrict__ gates, int64_t ldg, const float* __restrict__ lam,
                                          float* __restrict__ y, int64_t ldy, const float* __restrict__ y_bias, int64_t rows, int C, int n, float decay_scale) {
    pdl_wait();
    pdl_trigger();
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * C) return;
    const int64_t t = i / C;
    const int c = (int)(i - t * C);
    const int blk = c / n, j = c - blk * n;
    float* gr = gates + t * ldg + blk * 2 * n + j;
    const float la = -decay_scale * softplus_f(lam[c]) * sigmoid_f(gr[0]);
    const float b = sqrtf(-expm1f(2.0f * la)) * sigmoid_f(gr[n]) * u[t * ldu + c];
    gr[0] = expf(la);
    gr[n] = b;
    y[t * ldy + c] = gelu_tanh_f(y[t * ldy + c] + (y_bias ? y_bias[c] : 0.f));
}

template <typename TOut>
__global__ void __launch_bounds__(32)
linear_scan_kernel(const float* __restrict__ gates, int64_t ldg, const float* __restrict__ y, int64_t ldy, float* __restrict__ state, TOut* __restrict__ out,
                   const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ seq_slots, const int32_t* __restrict__ seq_start, int C, int n) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 32 + threadIdx.x;
    const int b = blockIdx.y;
    if (c >= C) return;
    const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
    if (t1 <= t0) return;
    float* sp = state + (int64_t)seq_slots[b] * C + c;
    float S = seq_start[b] == 0 ? 0.f : *sp;
    const int blk = c / n, j = c - blk * n;
    const float* ga = gates + blk * 2 * n + j;
    constexpr int kAhead = 16;
    float na[kAhead], nb[kAhead], ny[kAhead];
#pragma unroll
    for (int a = 0; a < kAhead; ++a) {
        const int64_t t = min(t0 + a, t1 - 1);
        na[a] = ga[t * ldg]; nb[a] = ga[t * ldg + n]; ny[a] = y[t * ldy + c];
    }
    for (int tb = t0; tb < t1; tb += kAhead) {
        float ca[kAhead], cb[kAhead], cy[kAhead];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) { ca[a] = na[a]; cb[a] = nb[a]; cy[a] = ny[a]; }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int64_t t = min(tb + kAhead + a, t1 - 1);
            na[a] = ga[t * ldg]; nb[a] = ga[t * ldg + n]; ny[a] = y[t * ldy + c];
        }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            if (tb + a >= t1) break;
            S = fmaf(ca[a], S, cb[a]);
            out[(int64_t)(tb + a) * C + c] = from_f32<TOut>(S * cy[a]);
        }
    }
    *sp = S;
}

// Long portions: the bare scan cut into chunks of 128 rows, all chunks at once.  A chunk's rows compose to S_out = P S_in + Q with P the product of
// its a_t and Q its own scan from zero: one kernel takes (P, Q) of every chunk, one walks an entry's chunks per channel and leaves every chunk's S_in,
// one replays every chunk from its S_in and writes the outputs.  The association of the sums differs from the row-by-row scan by rounding only.
constexpr int kScanChunk = 128;

__device__ __forceinline__ int scan_chunk_base(const int32_t* cu, int b) {
    int s = 0;
    for (int i = 0; i < b; ++i) s += (cu[i + 1] - cu[i] + kScanChunk - 1) / kScanChunk;
    return s;
}

__global__ void __launch_bounds__(128)
scan_chunk_compose_kernel(const float* __restrict__ gates, int64_t ldg, float* __restrict__ pq, const int32_t* __restrict__ cu_seqlens, int C, int n) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 128 + threadIdx.x, ch = blockIdx.y, b = blockIdx.z;
    if (c >= C) return;
    const int t0 = cu_seqlens[b], rows = cu_seqlens[b + 1] - t0;
    if (ch * kScanChunk >= rows) return;
    const int tf = t0 + ch * kScanChunk, nt = min(kScanChunk, rows - ch * kScanChunk);
    const int blk = c / n, j = c - blk * n;
    const float* ga = gates + (int64_t)tf * ldg + blk * 2 * n + j;
    float P = 1.f, Q = 0.f;
#pragma unroll 8
    for (int t = 0; t < nt; ++t) {
        const float a = ga[(int64_t)t * ldg], bb = ga[(int64_t)t * ldg + n];
        Q = fmaf(a, Q, bb);
        P *= a;
    }
    const int64_t at = ((int64_t)(scan_chunk_base(cu_seqlens, b) + ch) * C + c) * 2;
    pq[at] = P; pq[at + 1] = Q;
}

__global__ void __launch_bounds__(128)
scan_chunk_carry_kernel(float* __restrict__ pq, float* __restrict__ state, const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ seq_slots,
                        const int32_t* __restrict__ seq_start, int C) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
    if (c >= C) return;
    const int rows = cu_seqlens[b + 1] - cu_seqlens[b];
    if (rows <= 0) return;
    const int nc = (rows + kScanChunk - 1) / kScanChunk;
    float* sp = state + (int64_t)seq_slots[b] * C + c;
    float S = seq_start[b] == 0 ? 0.f : *sp;
    float2* p0 = reinterpret_cast<float2*>(pq) + (int64_t)scan_chunk_base(cu_seqlens, b) * C + c;
    constexpr int kAhead = 8;
    float2 nx[kAhead];
#pragma unroll
    for (int a = 0; a < kAhead; ++a) nx[a] = p0[(int64_t)min(a, nc - 1) * C];
    for (int cb = 0; cb < nc; cb += kAhead) {
        float2 cur[kAhead];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) cur[a] = nx[a];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) nx[a] = p0[(int64_t)min(cb + kAhead + a, nc - 1) * C];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            if (cb + a >= nc) break;
            p0[(int64_t)(cb + a) * C].y = S;                 // the state that enters the chunk
            S = fmaf(cur[a].x, S, cur[a].y);
        }
    }
    *sp = S;
}

template <typename TOut>
__global__ void __launch_bounds__(128)
scan_chunk_replay_kernel(const float* __restrict__ gates, int64_t ldg, const float* __restrict__ y, int64_t ldy, const float* __restrict__ pq, TOut* __restrict__ out,
                         const int32_t* __restrict__ cu_seqlens, int C, int n) {
    pdl_wait();
    pdl_trigger();
    const int c = blockIdx.x * 128 + threadIdx.x, ch = blockIdx.y, b = blockIdx.z;
    if (c >= C) return;
    const int t0 = cu_seqlens[b], rows = cu_seqlens[b + 1] - t0;
    if (ch * kScanChunk >= rows) return;
    const int tf = t0 + ch * kScanChunk, nt = min(kScanChunk, rows - ch * kScanChunk);
    const int blk = c / n, j = c - blk * n;
    const float* ga = gates + (int64_t)tf * ldg + blk * 2 * n + j;
    const float* yp = y + (int64_t)tf * ldy + c;
    TOut* op = out + (int64_t)tf * C + c;
    float S = pq[((int64_t)(scan_chunk_base(cu_seqlens, b) + ch) * C + c) * 2 + 1];
#pragma unroll 8
    for (int t = 0; t < nt; ++t) {
        S = fmaf(ga[(int64_t)t * ldg], S, ga[(int64_t)t * ldg + n]);
        op[(int64_t)t * C] = from_f32<TOut>(S * yp[(int64_t)t * ldy]);
    }
}

// ---- linear attention with a matrix state ---------------------------------------------------------------------------------------------
constexpr int kTile = 16;
constexpr int kScanChunkedRows = 512;    // entries with at least this many rows (and a scratch buffer): the bare scan runs over chunks of 128 rows, all at once
constexpr int kScanSplitRows = 16;     // entries with at least this many rows: the gated scan runs as a row-parallel pass plus a bare scan

struct LinAttnArgs {
    const float* proj; int64_t ld;
    int64_t off_q, off_k, off_v; int off_i, off_f;      // columns of proj: q, k [H dk], v [H dv], gate pre-activations [H] (exponential gating only)
    const float* decay;                          // [H] (fixed decay)
    const float* i_bias; const float* f_bias;    // [H]
    float cap, q_scale; int act;
    float* S; float* nrm; float* mx;             // [slots, H, dv, dk], [slots, H, ceil(dv / 16), dk], [slots, H, ceil(dv / 16)]
    float* out;                                  // [T, H dv]
    const int32_t* cu_seqlens; const int32_t* seq_slots; const int32_t* seq_start;
    int H, dk, dv;
    const float* alpha; int64_t lda;             // [T, H dk] row pitch lda: one decay per token and key row (channel decay)
    const float* bonus;                          // [H, dk]: the output is read before the token joins the state, which it enters with this weight (channel decay)
};

// kG: 0 = a fixed decay per head, 1 = exponential gating, 2 = a decay per key row and token, 3 = the same with the output read BEFORE the token's decay and
// write: o_t = (S_(t-1) + diag(bonus) k_t v_t^T)^T q_t
template <int kR, int kG>
__global__ void __launch_bounds__(128)
linear_attention_kernel(const LinAttnArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr bool kExp = kG == 1, kChan = kG >= 2, kBonus = kG == 3;
    constexpr int kP = 8 * kR;                   // padded key rows
    extern __shared__ __align__(16) float smem[];
    float* sq = smem;                            // [kTile][kP]
    float* sk = sq + kTile * kP;                 // [kTile][kP]
    float* sal = sk + kTile * kP;                // [kTile][kP] decays of the key rows (channel decay only)
    float* sv = sal + (kChan ? kTile * kP : 0);  // [kTile][16]
    float* sa = sv + kTile * 16;                 // [kTile] decay of the state
    float* sb = sa + kTile;                      // [kTile] weight of the new outer product
    float* se = sb + kTile;                      // [kTile] e^(-m_t)
    float* sf = se + kTile;                      // [kTile] f_t
    float* si = sf + kTile;                      // [kTile] i_t
    float* sm = si + kTile;                      // [kTile + 1] m before the tile's first token, then m_t
    const int h = blockIdx.y, b = blockIdx.z;
    const int H = A.H, dk = A.dk, dv = A.dv;
    const int t0 = A.cu_seqlens[b], t1 = A.cu_seqlens[b + 1];
    if (t1 <= t0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int part = lane >> 2, cl = lane & 3;
    const int colb = warp * 4 + cl;              // column inside the block's 16
    const int col = blockIdx.x * 16 + colb;
    const bool col_ok = col < dv;
    const bool fresh = A.seq_start[b] == 0;
    const int64_t slot = A.seq_slots[b];
    const bool vec = (dk & 3) == 0;              // a lane's rows of the state are then whole 16-byte words
    float* Sp = A.S + ((slot * H + h) * dv + (col_ok ? col : 0)) * (int64_t)dk + part * kR;
    // the normaliser and the maximum are kept once per block of 16 columns: every block reads and writes a copy of its own
    const int64_t own = (slot * H + h) * (int64_t)gridDim.x + blockIdx.x;
    float* np = kExp ? A.nrm + own * dk + part * kR : nullptr;
    float S[kR], nv[kR];
#pragma unroll
    for (int r = 0; r < kR; ++r) { S[r] = 0.f; nv[r] = 0.f; }
    if (!fresh) {
        if (vec) {
#pragma unroll
            for (int r4 = 0; r4 < kR / 4; ++r4) {
                if (part * kR + r4 * 4 >= dk) continue;
                if (col_ok) { const float4 v = reinterpret_cast<const float4*>(Sp)[r4]; S[r4 * 4] = v.x; S[r4 * 4 + 1] = v.y; S[r4 * 4 + 2] = v.z; S[r4 * 4 + 3] = v.w; }
                if (kExp) { const float4 v = reinterpret_cast<const float4*>(np)[r4]; nv[r4 * 4] = v.x; nv[r4 * 4 + 1] = v.y; nv[r4 * 4 + 2] = v.z; nv[r4 * 4 + 3] = v.w; }
            }
        } else {
#pragma unroll
            for (int r = 0; r < kR; ++r) {
                const bool ok = part * kR + r < dk;
                if (col_ok && ok) S[r] = Sp[r];
                if (kExp && ok) nv[r] = np[r];
            }
        }
    }
    if (kExp && threadIdx.x == 0) sm[0] = fresh ? 0.f : A.mx[own];
    const float fixed_a = kG == 0 ? A.decay[h] : 0.f;
    float bo[kBonus ? kR : 1];
    if (kBonus) {
#pragma unroll
        for (int r = 0; r < kR; ++r) bo[kBonus ? r : 0] = part * kR + r < dk ? A.bonus[h * dk + part * kR + r] : 0.f;
    }
    // the next tile's operands travel in registers while the current tile is walked: element e = thread + 128 i of the tile's [16][kP] q and k
    // rows, two of its [16][16] values, and (lanes 0..15 of the last warp) the two gate pre-activations of a token
    float pq[kR], pk[kR], pal[kChan ? kR : 1], pv[2], pgi = 0.f, pgf = 0.f;
    auto fetch = [&](int tb) {
        const int nt = min(kTile, t1 - tb);
#pragma unroll
        for (int i = 0; i < kR; ++i) {
            const int e = threadIdx.x + 128 * i, tt = e / kP, r = e - tt * kP;
            const bool ok = tt < nt && r < dk;
            const float* row = A.proj + (int64_t)(tb + (ok ? tt : 0)) * A.ld;
            pq[i] = ok ? row[A.off_q + h * dk + r] : 0.f;
            pk[i] = ok ? row[A.off_k + h * dk + r] : 0.f;
            if (kChan) pal[i] = ok ? A.alpha[(int64_t)(tb + tt) * A.lda + h * dk + r] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int e = threadIdx.x + 128 * i, tt = e >> 4, gc = blockIdx.x * 16 + (e & 15);
            pv[i] = (tt < nt && gc < dv) ? A.proj[(int64_t)(tb + tt) * A.ld + A.off_v + h * dv + gc] : 0.f;
        }
        if (kExp && warp == 3 && lane < nt) {
            const float* row = A.proj + (int64_t)(tb + lane) * A.ld;
            pgi = row[A.off_i + h] + (A.i_bias ? A.i_bias[h] : 0.f);
            pgf = row[A.off_f + h] + (A.f_bias ? A.f_bias[h] : 0.f);
        }
    };
    fetch(t0);
    for (int tb = t0; tb < t1; tb += kTile) {
        const int nt = min(kTile, t1 - tb);
        __syncthreads();                         // the previous tile has been walked
#pragma unroll
        for (int i = 0; i < kR; ++i) {
            const int e = threadIdx.x + 128 * i;
            float qv = pq[i], kv = pk[i];
            if (A.act == 1) { qv = silu_f(qv); kv = silu_f(kv); }
            sq[e] = qv * A.q_scale; sk[e] = kv;
            if (kChan) sal[e] = pal[i];
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) sv[threadIdx.x + 128 * i] = A.act == 1 ? silu_f(pv[i]) : pv[i];
        if (kExp && warp == 3) {
            // gate values of the tile's tokens, the chain of maxima, then the coefficients
            if (lane < nt) {
                si[lane] = A.cap * tanhf(pgi / A.cap);
                sf[lane] = log_sigmoid_f(A.cap * tanhf(pgf / A.cap));
            }
            __syncwarp();
            if (lane == 0) {
                float m = sm[0];
                for (int tt = 0; tt < nt; ++tt) { m = fmaxf(sf[tt] + m, si[tt]); sm[tt + 1] = m; }
            }
            __syncwarp();
            if (lane < nt) {
                const float m_prev = sm[lane], m_new = sm[lane + 1];
                sa[lane] = expf(sf[lane] + m_prev - m_new);
                sb[lane] = expf(si[lane] - m_new);
                se[lane] = expf(-m_new);
            }
        }
        __syncthreads();
        if (tb + kTile < t1) fetch(tb + kTile);
        // the tile's tokens one after the other; every token leaves a partial sum per lane, and the butterflies that join the eight parts run
        // afterwards for all tokens together (sixteen independent chains instead of one per token on the serial path)
        float osum[kTile], nsum[kTile];
#pragma unroll
        for (int tt = 0; tt < kTile; ++tt) {
            osum[tt] = 0.f; nsum[tt] = 0.f;
            if (tt >= nt) continue;
            const float a = kExp ? sa[tt] : fixed_a;
            const float bv = (kExp ? sb[tt] : 1.0f) * sv[tt * 16 + colb];
            const float bn = kExp ? sb[tt] : 0.f;
            float acc[2] = {0.f, 0.f}, nq[2] = {0.f, 0.f};
            const float4* q4 = reinterpret_cast<const float4*>(sq + tt * kP + part * kR);
            const float4* k4 = reinterpret_cast<const float4*>(sk + tt * kP + part * kR);
            const float4* a4 = reinterpret_cast<const float4*>(sal + tt * kP + part * kR);
#pragma unroll
            for (int r4 = 0; r4 < kR / 4; ++r4) {
                const float4 qq = q4[r4], kk = k4[r4], aa = kChan ? a4[r4] : make_float4(a, a, a, a);
                const float qa[4] = {qq.x, qq.y, qq.z, qq.w}, ka[4] = {kk.x, kk.y, kk.z, kk.w}, da[4] = {aa.x, aa.y, aa.z, aa.w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int r = r4 * 4 + j;
                    const float kv = ka[j] * bv;
                    if (kBonus) acc[j & 1] = fmaf(fmaf(bo[kBonus ? r : 0], kv, S[r]), qa[j], acc[j & 1]);
                    S[r] = fmaf(da[j], S[r], kv);
                    if (!kBonus) acc[j & 1] = fmaf(S[r], qa[j], acc[j & 1]);
                    if (kExp) { nv[r] = fmaf(a, nv[r], ka[j] * bn); nq[j & 1] = fmaf(nv[r], qa[j], nq[j & 1]); }
                }
            }
            osum[tt] = acc[0] + acc[1];
            if (kExp) nsum[tt] = nq[0] + nq[1];
        }
#pragma unroll
        for (int sh = 4; sh < 32; sh <<= 1) {
#pragma unroll
            for (int tt = 0; tt < kTile; ++tt) {
                osum[tt] += __shfl_xor_sync(0xffffffffu, osum[tt], sh);
                if (kExp) nsum[tt] += __shfl_xor_sync(0xffffffffu, nsum[tt], sh);
            }
        }
        if (part == 0 && col_ok) {
#pragma unroll
            for (int tt = 0; tt < kTile; ++tt) {
                if (tt >= nt) continue;
                float o = osum[tt];
                if (kExp) o = o / (fmaxf(fabsf(nsum[tt]), se[tt]) + 1e-6f);
                A.out[(int64_t)(tb + tt) * H * dv + h * dv + col] = o;
            }
        }
        if (kExp) {
            __syncthreads();
            if (threadIdx.x == 0) sm[0] = sm[nt];
        }
    }
    if (vec) {
#pragma unroll
        for (int r4 = 0; r4 < kR / 4; ++r4) {
            if (part * kR + r4 * 4 >= dk) continue;
            if (col_ok) reinterpret_cast<float4*>(Sp)[r4] = make_float4(S[r4 * 4], S[r4 * 4 + 1], S[r4 * 4 + 2], S[r4 * 4 + 3]);
            if (kExp && warp == 0 && cl == 0) reinterpret_cast<float4*>(np)[r4] = make_float4(nv[r4 * 4], nv[r4 * 4 + 1], nv[r4 * 4 + 2], nv[r4 * 4 + 3]);
        }
    } else {
#pragma unroll
        for (int r = 0; r < kR; ++r) {
            const bool ok = part * kR + r < dk;
            if (col_ok && ok) Sp[r] = S[r];
            if (kExp && ok && warp == 0 && cl == 0) np[r] = nv[r];
        }
    }
    if (kExp) {
        __syncthreads();
        if (threadIdx.x == 0) A.mx[own] = sm[0];
    }
}

// Steps in which every entry brings one token (row b belongs to entry b): nothing is staged and no thread waits for another -- a lane reads its
// own rows of q and k, its column's value and (exponential gating) the two gate values straight from the projection, takes one pass over its
// rows of the state and writes them back.  Same lane layout and state layout as the kernel above.
template <int kR, int kG>
__global__ void __launch_bounds__(128)
linear_attention_step_kernel(const LinAttnArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr bool kExp = kG == 1, kChan = kG >= 2, kBonus = kG == 3;
    const int h = blockIdx.y, b = blockIdx.z;
    const int H = A.H, dk = A.dk, dv = A.dv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int part = lane >> 2, cl = lane & 3;
    const int col = blockIdx.x * 16 + warp * 4 + cl;
    const bool col_ok = col < dv;
    const bool fresh = A.seq_start[b] == 0;
    const int64_t slot = A.seq_slots[b];
    const bool vec = (dk & 3) == 0;
    float* Sp = A.S + ((slot * H + h) * dv + (col_ok ? col : 0)) * (int64_t)dk + part * kR;
    const int64_t own = (slot * H + h) * (int64_t)gridDim.x + blockIdx.x;
    float* np = kExp ? A.nrm + own * dk + part * kR : nullptr;
    const float* row = A.proj + (int64_t)b * A.ld;
    float S[kR], nv[kR], q[kR], k[kR], al[kChan ? kR : 1];
#pragma unroll
    for (int r = 0; r < kR; ++r) {
        const int g = part * kR + r;
        const bool ok = g < dk;
        S[r] = 0.f; nv[r] = 0.f;
        q[r] = ok ? row[A.off_q + h * dk + g] : 0.f;
        k[r] = ok ? row[A.off_k + h * dk + g] : 0.f;
        if (kChan) al[r] = ok ? A.alpha[(int64_t)b * A.lda + h * dk + g] : 0.f;
    }
    float v = col_ok ? row[A.off_v + h * dv + col] : 0.f;
    float zi = 0.f, zf = 0.f, m_prev = 0.f;
    if (kExp) {
        zi = row[A.off_i + h] + (A.i_bias ? A.i_bias[h] : 0.f);
        zf = row[A.off_f + h] + (A.f_bias ? A.f_bias[h] : 0.f);
        if (!fresh) m_prev = A.mx[own];
    }
    if (!fresh) {
        if (vec) {
#pragma unroll
            for (int r4 = 0; r4 < kR / 4; ++r4) {
                if (part * kR + r4 * 4 >= dk) continue;
                if (col_ok) { const float4 t = reinterpret_cast<const float4*>(Sp)[r4]; S[r4 * 4] = t.x; S[r4 * 4 + 1] = t.y; S[r4 * 4 + 2] = t.z; S[r4 * 4 + 3] = t.w; }
                if (kExp) { const float4 t = reinterpret_cast<const float4*>(np)[r4]; nv[r4 * 4] = t.x; nv[r4 * 4 + 1] = t.y; nv[r4 * 4 + 2] = t.z; nv[r4 * 4 + 3] = t.w; }
            }
        } else {
#pragma unroll
            for (int r = 0; r < kR; ++r) {
                const bool ok = part * kR + r < dk;
                if (col_ok && ok) S[r] = Sp[r];
                if (kExp && ok) nv[r] = np[r];
            }
        }
    }
    float a = kG == 0 ? A.decay[h] : 0.f, bw = 1.0f, em = 0.f, m_new = 0.f;
    if (kExp) {
        const float gi = A.cap * tanhf(zi / A.cap), gf = log_sigmoid_f(A.cap * tanhf(zf / A.cap));
        m_new = fmaxf(gf + m_prev, gi);
        a = expf(gf + m_prev - m_new); bw = expf(gi - m_new); em = expf(-m_new);
    }
    if (A.act == 1) v = silu_f(v);
    const float bv = bw * v;
    float acc[2] = {0.f, 0.f}, nq[2] = {0.f, 0.f};
#pragma unroll
    for (int r = 0; r < kR; ++r) {
        float qv = q[r], kv = k[r];
        if (A.act == 1) { qv = silu_f(qv); kv = silu_f(kv); }
        qv *= A.q_scale;
        const float kvv = kv * bv;
        if (kBonus) acc[r & 1] = fmaf(fmaf(part * kR + r < dk ? A.bonus[h * dk + part * kR + r] : 0.f, kvv, S[r]), qv, acc[r & 1]);
        S[r] = fmaf(kChan ? al[kChan ? r : 0] : a, S[r], kvv);
        if (!kBonus) acc[r & 1] = fmaf(S[r], qv, acc[r & 1]);
        if (kExp) { nv[r] = fmaf(a, nv[r], kv * bw); nq[r & 1] = fmaf(nv[r], qv, nq[r & 1]); }
    }
    float o = acc[0] + acc[1], nqs = nq[0] + nq[1];
#pragma unroll
    for (int sh = 4; sh < 32; sh <<= 1) {
        o += __shfl_xor_sync(0xffffffffu, o, sh);
        if (kExp) nqs += __shfl_xor_sync(0xffffffffu, nqs, sh);
    }
    if (part == 0 && col_ok) {
        if (kExp) o = o / (fmaxf(fabsf(nqs), em) + 1e-6f);
        A.out[(int64_t)b * H * dv + h * dv + col] = o;
    }
    if (vec) {
#pragma unroll
        for (int r4 = 0; r4 < kR / 4; ++r4) {
            if (part * kR + r4 * 4 >= dk) continue;
            if (col_ok) reinterpret_cast<float4*>(Sp)[r4] = make_float4(S[r4 * 4], S[r4 * 4 + 1], S[r4 * 4 + 2], S[r4 * 4 + 3]);
            if (kExp && warp == 0 && cl == 0) reinterpret_cast<float4*>(np)[r4] = make_float4(nv[r4 * 4], nv[r4 * 4 + 1], nv[r4 * 4 + 2], nv[r4 * 4 + 3]);
        }
    } else {
#pragma unroll
        for (int r = 0; r < kR; ++r) {
            const bool ok = part * kR + r < dk;
            if (col_ok && ok) Sp[r] = S[r];
            if (kExp && ok && warp == 0 && cl == 0) np[r] = nv[r];
        }
    }
    if (kExp && threadIdx.x == 0) A.mx[own] = m_new;
}

// ---- portions of prompts: the same recurrence over chunks of 64 tokens, all chunks at once -----------------------------------------------------
// With F_t the sum of the log decays from the chunk's first token to t, li_t the log input weight and m_t the running maximum (F_t = (t + 1) ln decay,
// li = 0, m = 0 for a fixed decay), token t of a chunk that is entered with the (stabilised) state S_in and maximum m_in returns
//     o_t = e^(F_t + m_in - m_t) S_in^T q_t + sum_{j <= t} e^(F_t - F_j + li_j - m_t) (q_t . k_j) v_j
// and the chunk leaves  S_out = e^(F_L + m_in - m_L) S_in + sum_j e^(F_L - F_j + li_j - m_L) k_j v_j^T  (the normaliser alike, with k_j alone).  So:
//   la_gate_values   (exponential gating) log gates of every token, all rows at once;
//   la_gate_chain    per (entry, head) the chain of maxima m_t, exactly as the token-by-token kernel takes it, and F_t;
//   la_chunk_state   per chunk the second term of S_out, a [dv, dk] product over the chunk's tokens, all chunks at once;
//   la_chunk_scan    per state element the walk over an entry's chunks that turns those terms into the state entering every chunk (in place);
//   la_chunk_output  per chunk the two terms of o_t: scores against the chunk's own keys, then values and entering state in one accumulation.
// All arithmetic is f32 on the FMA pipe; the results differ from the token-by-token kernel by rounding only.
constexpr int kChunk = 64;

struct ChunkArgs {
    LinAttnArgs A;
    float* gc;            // [T, H, 3]: F_t, li_t, m_t (exponential gating)
    float* U;             // [chunk slots, H, dv, dk]
    float* un;            // [chunk slots, H, dk] a chunk's own term of the normaliser; with channel decay the product of the chunk's decays per key row
    float* un_in;         // [chunk slots, H, dk] the normaliser that enters the chunk
    float* m0;            // [entries, H] the maximum every entry starts this step with (the slot's copy changes while the kernels run)
    int max_chunks;       // the most chunks any entry has
    int gating;           // 0 fixed decay, 1 exponential, 2 channel decay
};

__device__ __forceinline__ int chunk_base(const int32_t* cu, int b) {      // chunk slots of the entries before b
    int s = 0;
    for (int i = 0; i < b; ++i) s += (cu[i + 1] - cu[i] + kChunk - 1) / kChunk;
    return s;
}
__device__ __forceinline__ float log_decay(float d) { return fmaxf(logf(d), -80.f); }

__global__ void la_gate_values_kernel(const ChunkArgs C, int T) {
    pdl_wait();
    pdl_trigger();
    const LinAttnArgs& A = C.A;
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= T * A.H) return;
    const int t = i / A.H, h = i - t * A.H;
    const float* row = A.proj + (int64_t)t * A.ld;
    const float zi = row[A.off_i + h] + (A.i_bias ? A.i_bias[h] : 0.f), zf = row[A.off_f + h] + (A.f_bias ? A.f_bias[h] : 0.f);
    C.gc[(int64_t)i * 3 + 1] = A.cap * tanhf(zi / A.cap);
    C.gc[(int64_t)i * 3 + 0] = log_sigmoid_f(A.cap * tanhf(zf / A.cap));
}

__global__ void la_gate_chain_kernel(const ChunkArgs C) {
    pdl_wait();
    pdl_trigger();
    const LinAttnArgs& A = C.A;
    const int h = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
    if (h >= A.H) return;
    const int t0 = A.cu_seqlens[b], t1 = A.cu_seqlens[b + 1];
    if (t1 <= t0) return;
    const int nvb = (A.dv + 15) / 16;
    float m = A.seq_start[b] == 0 ? 0.f : A.mx[((int64_t)A.seq_slots[b] * A.H + h) * nvb];
    C.m0[(int64_t)b * A.H + h] = m;
    float F = 0.f;
    // the chain itself is an add and a maximum per token; the log gates of the next sixteen tokens are in flight meanwhile
    constexpr int kAhead = 16;
    float nf[kAhead], ni[kAhead];
    float* g0 = C.gc + (int64_t)h * 3;
    const int64_t pitch = (int64_t)A.H * 3;
#pragma unroll
    for (int a = 0; a < kAhead; ++a) { const int64_t t = min(t0 + a, t1 - 1); nf[a] = g0[t * pitch]; ni[a] = g0[t * pitch + 1]; }
    for (int tb = t0; tb < t1; tb += kAhead) {
        float cf[kAhead], ci[kAhead];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) { cf[a] = nf[a]; ci[a] = ni[a]; }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) { const int64_t t = min(tb + kAhead + a, t1 - 1); nf[a] = g0[t * pitch]; ni[a] = g0[t * pitch + 1]; }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int t = tb + a;
            if (t >= t1) break;
            if ((t - t0) % kChunk == 0) F = 0.f;
            F += cf[a];
            m = fmaxf(cf[a] + m, ci[a]);
            g0[(int64_t)t * pitch] = F; g0[(int64_t)t * pitch + 2] = m;
        }
    }
}

// F, li, m of row t (tt = its index inside the chunk)
__device__ __forceinline__ void token_gate(const ChunkArgs& C, int h, int t, int tt, float lnd, float& F, float& li, float& m) {
    if (C.gating != 1) { F = (float)(tt + 1) * lnd; li = 0.f; m = 0.f; return; }
    const float* g = C.gc + ((int64_t)t * C.A.H + h) * 3;
    F = g[0]; li = g[1]; m = g[2];
}
__device__ __forceinline__ float chunk_m_in(const ChunkArgs& C, int b, int h, int t_first, int c) {
    if (C.gating != 1) return 0.f;
    if (c > 0) return C.gc[((int64_t)(t_first - 1) * C.A.H + h) * 3 + 2];
    return C.m0[(int64_t)b * C.A.H + h];
}

// U[slot, h, cv, r] = sum_j w_j v_j[cv] k_j[r], w_j = e^(F_L - F_j + li_j - m_L); a block makes a 64 x 64 tile, a thread 4 x 4 of it
__global__ void __launch_bounds__(256)
la_chunk_state_kernel(const ChunkArgs C) {
    pdl_wait();
    pdl_trigger();
    const LinAttnArgs& A = C.A;
    __shared__ __align__(16) float vs[kChunk][64 + 4], ks[kChunk][64 + 4];          // rows of 68 floats: 16-byte reads of four neighbours
    __shared__ float ws[kChunk];
    const int h = blockIdx.y, b = blockIdx.z / C.max_chunks, c = blockIdx.z % C.max_chunks;
    const int t0 = A.cu_seqlens[b], rows = A.cu_seqlens[b + 1] - t0;
    if (c * kChunk >= rows) return;
    const int tf = t0 + c * kChunk, nt = min(kChunk, rows - c * kChunk);
    const int dk = A.dk, dv = A.dv, H = A.H;
    const int tiles_r = (dk + 63) / 64;
    const int cv0 = (blockIdx.x / tiles_r) * 64, r0 = (blockIdx.x % tiles_r) * 64;
    const int slot = chunk_base(A.cu_seqlens, b) + c;
    const float lnd = C.gating == 0 ? log_decay(A.decay[h]) : 0.f;
    if (threadIdx.x < kChunk) {
        float w = 0.f;
        if ((int)threadIdx.x < nt) {
            float F, li, m, FL, liL, mL;
            token_gate(C, h, tf + threadIdx.x, threadIdx.x, lnd, F, li, m);
            token_gate(C, h, tf + nt - 1, nt - 1, lnd, FL, liL, mL);
            w = expf(FL - F + li - mL);
        }
        ws[threadIdx.x] = w;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < kChunk * 64; e += 256) {
        const int j = e >> 6, x = e & 63;
        float v = 0.f, k = 0.f;
        if (j < nt) {
            const float* row = A.proj + (int64_t)(tf + j) * A.ld;
            if (cv0 + x < dv) { v = row[A.off_v + h * dv + cv0 + x]; if (A.act == 1) v = silu_f(v); }
            if (r0 + x < dk) { k = row[A.off_k + h * dk + r0 + x]; if (A.act == 1) k = silu_f(k); }
        }
        vs[j][x] = v * ws[j]; ks[j][x] = k;
    }
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int j = 0; j < nt; ++j) {
        const float4 a4 = *reinterpret_cast<const float4*>(&vs[j][ty * 4]), k4 = *reinterpret_cast<const float4*>(&ks[j][tx * 4]);
        const float a[4] = {a4.x, a4.y, a4.z, a4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int l = 0; l < 4; ++l) acc[i][l] = fmaf(a[i], k[l], acc[i][l]);
    }
    float* U = C.U + ((int64_t)slot * H + h) * dv * dk;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int cv = cv0 + ty * 4 + i;
        if (cv >= dv) continue;
#pragma unroll
        for (int l = 0; l < 4; ++l) {
            const int r = r0 + tx * 4 + l;
            if (r < dk) U[(int64_t)cv * dk + r] = acc[i][l];
        }
    }
    if (C.gating == 1 && cv0 == 0 && threadIdx.x < 64 && r0 + (int)threadIdx.x < dk) {
        float s = 0.f;
        for (int j = 0; j < nt; ++j) s = fmaf(ws[j], ks[j][threadIdx.x], s);
        C.un[((int64_t)slot * H + h) * dk + r0 + threadIdx.x] = s;
    }
}

// a thread owns one state element (h, cv, r): U[c] <- the state that enters chunk c, the state slot <- the state after the last chunk
__global__ void __launch_bounds__(256)
la_chunk_scan_kernel(const ChunkArgs C) {
    pdl_wait();
    pdl_trigger();
    const LinAttnArgs& A = C.A;
    const int b = blockIdx.y;
    const int dk = A.dk, dv = A.dv, H = A.H;
    const int64_t e = (int64_t)blockIdx.x * 256 + threadIdx.x;
    if (e >= (int64_t)H * dv * dk) return;
    const int h = (int)(e / ((int64_t)dv * dk));
    const int cv = (int)((e / dk) % dv), r = (int)(e % dk);
    const int t0 = A.cu_seqlens[b], rows = A.cu_seqlens[b + 1] - t0;
    if (rows <= 0) return;
    const int nc = (rows + kChunk - 1) / kChunk;
    const int base = chunk_base(A.cu_seqlens, b);
    const bool fresh = A.seq_start[b] == 0;
    const int64_t slot = A.seq_slots[b];
    const int nvb = (dv + 15) / 16;
    float* Sp = A.S + ((slot * H + h) * dv + cv) * (int64_t)dk + r;
    const bool carries_n = C.gating == 1 && (cv & 15) == 0;            // one copy of the normaliser and of the maximum per 16 value columns
    float* np = carries_n ? A.nrm + ((slot * H + h) * nvb + (cv >> 4)) * (int64_t)dk + r : nullptr;
    float S = fresh ? 0.f : *Sp;
    float n = (carries_n && !fresh) ? *np : 0.f;
    const float lnd = C.gating == 0 ? log_decay(A.decay[h]) : 0.f;
    float m_in = chunk_m_in(C, b, h, t0, 0);
    // a chunk's term does not depend on the walk: the terms of the next eight chunks are in flight while the current one is applied
    constexpr int kAhead = 8;
    const int64_t ustride = (int64_t)H * dv * dk, nstride = (int64_t)H * dk;
    float* u0 = C.U + (((int64_t)base * H + h) * dv + cv) * dk + r;
    const int64_t n0 = ((int64_t)base * H + h) * dk + r;
    float nu[kAhead], nn[kAhead];
#pragma unroll
    for (int a = 0; a < kAhead; ++a) {
        const int c = min(a, nc - 1);
        nu[a] = u0[c * ustride];
        nn[a] = (carries_n || C.gating == 2) ? C.un[n0 + c * nstride] : 0.f;      // channel decay: the product of the chunk's decays of this key row
    }
    for (int cb = 0; cb < nc; cb += kAhead) {
        float cu[kAhead], cn[kAhead];
#pragma unroll
        for (int a = 0; a < kAhead; ++a) { cu[a] = nu[a]; cn[a] = nn[a]; }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int c = min(cb + kAhead + a, nc - 1);
            nu[a] = u0[c * ustride];
            nn[a] = (carries_n || C.gating == 2) ? C.un[n0 + c * nstride] : 0.f;
        }
#pragma unroll
        for (int a = 0; a < kAhead; ++a) {
            const int c = cb + a;
            if (c >= nc) break;
            const int nt = min(kChunk, rows - c * kChunk);
            float FL, liL, mL;
            token_gate(C, h, t0 + c * kChunk + nt - 1, nt - 1, lnd, FL, liL, mL);
            const float g = C.gating == 2 ? cn[a] : expf(FL + m_in - mL);
            u0[c * ustride] = S;
            S = fmaf(g, S, cu[a]);
            if (carries_n) {
                if (cv == 0) C.un_in[n0 + c * nstride] = n;               // the output kernel reads the entering normaliser from here
                n = fmaf(g, n, cn[a]);
            }
            m_in = mL;
        }
    }
    *Sp = S;
    if (carries_n) {
        *np = n;
        if (r == 0) A.mx[(slot * H + h) * nvb + (cv >> 4)] = m_in;
    }
}

// o for the 64 tokens of a chunk and 64 value columns: scores against the chunk's own keys, weights, then values and entering state
__global__ void __launch_bounds__(256, 3)
la_chunk_output_kernel(const ChunkArgs C) {
    pdl_wait();
    pdl_trigger();
    const LinAttnArgs& A = C.A;
    extern __shared__ __align__(16) float sm[];
    // every tile is stored so that the four neighbours a thread multiplies together are one 16-byte read (rows of 68 floats)
    float (*qs)[68] = reinterpret_cast<float (*)[68]>(sm);                          // [32][68] a slab of 32 key rows of q: [key row][token]
    float (*ks)[68] = reinterpret_cast<float (*)[68]>(sm + 32 * 68);                // [32][68] the same slab of k: [key row][token]; later of the entering state
    float (*pw)[68] = reinterpret_cast<float (*)[68]>(sm + 2 * 32 * 68);            // [64][68] weighted scores: [key token j][query token t]
    float (*vs)[68] = reinterpret_cast<float (*)[68]>(sm + 2 * 32 * 68 + 64 * 68);  // [64][68] values: [token][column]
    float* sF = sm + 2 * 32 * 68 + 2 * 64 * 68;                                     // [64] F_t, li_t, m_t, c_t, n_in . q_t
    float* sL = sF + 64; float* sM = sL + 64; float* sC = sM + 64; float* sN = sC + 64;
    const int h = blockIdx.y, b = blockIdx.z / C.max_chunks, c = blockIdx.z % C.max_chunks;
    const int t0 = A.cu_seqlens[b], rows = A.cu_seqlens[b + 1] - t0;
    if (c * kChunk >= rows) return;
    const int tf = t0 + c * kChunk, nt = min(kChunk, rows - c * kChunk);
    const int dk = A.dk, dv = A.dv, H = A.H;
    const int cv0 = blockIdx.x * 64;
    const int slot = chunk_base(A.cu_seqlens, b) + c;
    const float lnd = C.gating == 0 ? log_decay(A.decay[h]) : 0.f;
    const float m_in = chunk_m_in(C, b, h, tf, c);
    const float* Uin = C.U + ((int64_t)slot * H + h) * dv * dk;
    const float* nin = C.un_in + ((int64_t)slot * H + h) * dk;
    if (threadIdx.x < 64) {
        float F = 0.f, li = 0.f, m = 0.f, nq = 0.f;
        if ((int)threadIdx.x < nt) {
            token_gate(C, h, tf + threadIdx.x, threadIdx.x, lnd, F, li, m);
            if (C.gating == 1) {
                const float* row = A.proj + (int64_t)(tf + threadIdx.x) * A.ld + A.off_q + h * dk;
                for (int r = 0; r < dk; ++r) nq = fmaf(nin[r], (A.act == 1 ? silu_f(row[r]) : row[r]) * A.q_scale, nq);
            }
        }
        sF[threadIdx.x] = F; sL[threadIdx.x] = li; sM[threadIdx.x] = m; sC[threadIdx.x] = expf(F + m_in - m); sN[threadIdx.x] = nq;
    }
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    // a thread's eight elements of a 64 x 32 slab: (j, x) = (e >> 5, e & 31), e = thread + 256 i.  The next slab's elements are fetched into registers
    // before the current slab is multiplied, so that the loads are in flight during the products.
    float rq[8], rk[8];
    auto fetch_qk = [&](int r0, bool with_k) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i, j = e >> 5, x = e & 31;
            const bool ok = j < nt && r0 + x < dk;
            const float* row = A.proj + (int64_t)(tf + (ok ? j : 0)) * A.ld;
            rq[i] = ok ? row[A.off_q + h * dk + r0 + x] : 0.f;
            if (with_k) rk[i] = ok ? row[A.off_k + h * dk + r0 + x] : 0.f;
        }
    };
    // scores: rows ty * 4 .., keys tx * 4 ..
    fetch_qk(0, true);
    for (int r0 = 0; r0 < dk; r0 += 32) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i, j = e >> 5, x = e & 31;
            float q = rq[i], k = rk[i];
            if (A.act == 1) { q = silu_f(q); k = silu_f(k); }
            qs[x][j] = q * A.q_scale; ks[x][j] = k;
        }
        __syncthreads();
        if (r0 + 32 < dk) fetch_qk(r0 + 32, true);
#pragma unroll 8
        for (int x = 0; x < 32; ++x) {
            const float4 a4 = *reinterpret_cast<const float4*>(&qs[x][ty * 4]), k4 = *reinterpret_cast<const float4*>(&ks[x][tx * 4]);
            const float a[4] = {a4.x, a4.y, a4.z, a4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int l = 0; l < 4; ++l) acc[i][l] = fmaf(a[i], k[l], acc[i][l]);
        }
    }
    // the values of the chunk travel while the weights are worked out
    float rv[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int e = threadIdx.x + 256 * i, j = e >> 6, x = e & 63;
        rv[i] = (j < nt && cv0 + x < dv) ? A.proj[(int64_t)(tf + j) * A.ld + A.off_v + h * dv + cv0 + x] : 0.f;
    }
#pragma unroll
    for (int l = 0; l < 4; ++l) {
        const int j = tx * 4 + l;
        float w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int t = ty * 4 + i;
            w[i] = (j <= t && t < nt) ? acc[i][l] * expf(sF[t] - sF[j] + sL[j] - sM[t]) : 0.f;
        }
        *reinterpret_cast<float4*>(&pw[j][ty * 4]) = make_float4(w[0], w[1], w[2], w[3]);
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int e = threadIdx.x + 256 * i;
        vs[e >> 6][e & 63] = A.act == 1 ? silu_f(rv[i]) : rv[i];
    }
    __syncthreads();
    // the first slab of q and of the entering state for the second term travels during the first term's products
    float ru[8];
    auto fetch_u = [&](int r0) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i, j = e >> 5, x = e & 31;
            ru[i] = (cv0 + j < dv && r0 + x < dk) ? Uin[(int64_t)(cv0 + j) * dk + r0 + x] : 0.f;
        }
    };
    fetch_qk(0, false);
    fetch_u(0);
    // first term of the output: weighted scores times values (rows ty * 4 .., columns tx * 4 ..)
    float o1[4][4] = {}, o2[4][4] = {};
    for (int j = 0; j < nt; ++j) {
        const float4 p4 = *reinterpret_cast<const float4*>(&pw[j][ty * 4]), v4 = *reinterpret_cast<const float4*>(&vs[j][tx * 4]);
        const float p[4] = {p4.x, p4.y, p4.z, p4.w}, v[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int l = 0; l < 4; ++l) o1[i][l] = fmaf(p[i], v[l], o1[i][l]);
    }
    // second term: q against the state that entered the chunk, a slab of 32 key rows at a time
    float (*ss)[68] = ks;                                                           // [32][68] the entering state: [key row][column], over the k slab
    for (int r0 = 0; r0 < dk; r0 += 32) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i, j = e >> 5, x = e & 31;
            qs[x][j] = (A.act == 1 ? silu_f(rq[i]) : rq[i]) * A.q_scale;
            ss[x][j] = ru[i];                        // the same index pair read the other way: column j of the tile, key row x
        }
        __syncthreads();
        if (r0 + 32 < dk) { fetch_qk(r0 + 32, false); fetch_u(r0 + 32); }
#pragma unroll 8
        for (int x = 0; x < 32; ++x) {
            const float4 a4 = *reinterpret_cast<const float4*>(&qs[x][ty * 4]), u4 = *reinterpret_cast<const float4*>(&ss[x][tx * 4]);
            const float a[4] = {a4.x, a4.y, a4.z, a4.w}, u[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int l = 0; l < 4; ++l) o2[i][l] = fmaf(a[i], u[l], o2[i][l]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty * 4 + i;
        if (t >= nt) continue;
        float den = 1.0f;
        if (C.gating == 1) {
            float nq = sC[t] * sN[t];
            for (int j = 0; j <= t; ++j) nq += pw[j][t];
            den = fmaxf(fabsf(nq), expf(-sM[t])) + 1e-6f;
        }
#pragma unroll
        for (int l = 0; l < 4; ++l) {
            const int cv = cv0 + tx * 4 + l;
            if (cv < dv) A.out[(int64_t)(tf + t) * H * dv + h * dv + cv] = fmaf(sC[t], o2[i][l], o1[i][l]) / den;
        }
    }
}

// ---- a decay per token and key row (gated linear attention) over chunks --------------------------------------------------------------------------
// S_t = diag(a_t) S_(t-1) + k_t v_t^T.  Everything is built from PRODUCTS of decays, all of them in [0, 1], so nothing overflows whatever the decays are
// and a product that underflows is a contribution that has died.  With tokens grouped in runs of four, run c's product E_c, the product P_t of a
// token's own run up to and including t and the product R_j of a token's own run after j:
//     chunk state term     sum_j (prod_{i > j} a_i * k_j) v_j^T                                       (la_chan_state_kernel; E of the whole chunk beside it)
//     score of t over j    sum_r q_t P_t (prod_{runs between} E) R_j k_j, j in an earlier run; inside one run the products of at most three decays
//     entering state       q_t P_t prod_{runs before} E against S_in                                      (la_chan_output_kernel)
// The walk over the chunks is la_chunk_scan_kernel with the chunk's product per key row in place of the scalar decay.
// what becomes of z = w y + bias: 0 = sigmoid(z)^(1 / tau); 1 = exp(-exp(z)); 2 = exp(-exp(log_rate) softplus(z)); 3 = z itself
__device__ __forceinline__ float low_rank_value(float z, int form, float inv_tau, float log_rate) {
    if (form == 0) return expf(log_sigmoid_f(z) * inv_tau);
    if (form == 1) return expf(-expf(z));
    if (form == 2) return expf(-expf(log_rate) * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
    return z;
}

// few rows: 32 channels x 32 tokens per block (a lane per channel, a warp per four tokens), 64 inner values at a time through shared memory
__global__ void __launch_bounds__(256)
low_rank_rows_kernel(const float* __restrict__ y, int64_t ldy, const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ out, int T, int N,
                     int R, float inv_tau, int in_tanh, int form, const float* __restrict__ log_rate, int channels_per_rate) {
    pdl_wait();
    pdl_trigger();
    constexpr int kS = 64, kP = kS + 4;
    __shared__ __align__(16) float ws[32][kP], ys[32][kP];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int n0 = blockIdx.x * 32, n = n0 + lane, t0 = blockIdx.y * 32;
    float z[4];
    const float b = (n < N && bias) ? bias[n] : 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) z[i] = b;
    float rw[8], ry[8];
    auto fetch = [&](int r0) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i, j = e >> 6, r = r0 + (e & 63);
            rw[i] = (n0 + j < N && r < R) ? w[(int64_t)(n0 + j) * R + r] : 0.f;
            ry[i] = (t0 + j < T && r < R) ? y[(int64_t)(t0 + j) * ldy + r] : 0.f;
        }
    };
    fetch(0);
    for (int r0 = 0; r0 < R; r0 += kS) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i;
            ws[e >> 6][e & 63] = rw[i];
            ys[e >> 6][e & 63] = in_tanh ? tanhf(ry[i]) : ry[i];
        }
        __syncthreads();
        if (r0 + kS < R) fetch(r0 + kS);
        if (t0 + warp * 4 >= T) continue;
#pragma unroll 4
        for (int r = 0; r < kS; r += 4) {
            const float4 v = *reinterpret_cast<const float4*>(&ws[lane][r]);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float4 q = *reinterpret_cast<const float4*>(&ys[warp * 4 + i][r]);
                z[i] = fmaf(v.x, q.x, fmaf(v.y, q.y, fmaf(v.z, q.z, fmaf(v.w, q.w, z[i]))));
            }
        }
    }
    if (n >= N) return;
    const float lr = form == 2 ? log_rate[n / channels_per_rate] : 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i)
        if (t0 + warp * 4 + i < T) out[(int64_t)(t0 + warp * 4 + i) * N + n] = low_rank_value(z[i], form, inv_tau, lr);
}

// many rows: tiles of 64 tokens x 128 channels, 16 inner values at a time through shared memory (both operands stored inner value first), a thread makes 8 tokens x 4
// neighbouring channels
__global__ void __launch_bounds__(256)
low_rank_tile_kernel(const float* __restrict__ y, int64_t ldy, const float* __restrict__ w, const float* __restrict__ bias, float* __restrict__ out, int T, int N,
                     int R, float inv_tau, int in_tanh, int form, const float* __restrict__ log_rate, int channels_per_rate) {
    pdl_wait();
    pdl_trigger();
    __shared__ __align__(16) float ys[16][64 + 4], ws[16][128 + 4];
    const int n0 = blockIdx.x * 128, t0 = blockIdx.y * 64;
    const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5;
    float acc[8][4], ry[4], rw[8];
#pragma unroll
    for (int l = 0; l < 4; ++l) {
        const int n = n0 + tx * 4 + l;
        const float b = (n < N && bias) ? bias[n] : 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[i][l] = b;
    }
    auto fetch = [&](int r0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = threadIdx.x + 256 * i, t = e >> 4, r = e & 15;
            ry[i] = (t0 + t < T && r0 + r < R) ? y[(int64_t)(t0 + t) * ldy + r0 + r] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i, n = e >> 4, r = e & 15;
            rw[i] = (n0 + n < N && r0 + r < R) ? w[(int64_t)(n0 + n) * R + r0 + r] : 0.f;
        }
    };
    fetch(0);
    for (int r0 = 0; r0 < R; r0 += 16) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 4; ++i) { const int e = threadIdx.x + 256 * i; ys[e & 15][e >> 4] = in_tanh ? tanhf(ry[i]) : ry[i]; }
#pragma unroll
        for (int i = 0; i < 8; ++i) { const int e = threadIdx.x + 256 * i; ws[e & 15][e >> 4] = rw[i]; }
        __syncthreads();
        if (r0 + 16 < R) fetch(r0 + 16);
#pragma unroll
        for (int r = 0; r < 16; ++r) {
            const float4 a = *reinterpret_cast<const float4*>(&ys[r][ty * 8]), b = *reinterpret_cast<const float4*>(&ys[r][ty * 8 + 4]),
                         v = *reinterpret_cast<const float4*>(&ws[r][tx * 4]);
            const float yv[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w}, wv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int l = 0; l < 4; ++l) acc[i][l] = fmaf(wv[l], yv[i], acc[i][l]);
        }
    }
    float lr[4];
#pragma unroll
    for (int l = 0; l < 4; ++l) lr[l] = form == 2 && n0 + tx * 4 + l < N ? log_rate[(n0 + tx * 4 + l) / channels_per_rate] : 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = t0 + ty * 8 + i, n = n0 + tx * 4;
        if (t >= T || n >= N) continue;
        float o[4];
#pragma unroll
        for (int l = 0; l < 4; ++l) o[l] = low_rank_value(acc[i][l], form, inv_tau, lr[l]);
        float* dst = out + (int64_t)t * N + n;
        if (N % 4 == 0) { *reinterpret_cast<float4*>(dst) = make_float4(o[0], o[1], o[2], o[3]); continue; }
#pragma unroll
        for (int l = 0; l < 4; ++l)
            if (n + l < N) dst[l] = o[l];
    }
}

__global__ void __launch_bounds__(256)
la_chan_state_kernel(const ChunkArgs C) {
    pdl_wait();
    pdl_trigger();
    const LinAttnArgs& A = C.A;
    __shared__ __align__(16) float vs[kChunk][64 + 4], ks[kChunk][64 + 4];
    __shared__ float es[4][64];
    const int h = blockIdx.y, b = blockIdx.z / C.max_chunks, c = blockIdx.z % C.max_chunks;
    const int t0 = A.cu_seqlens[b], rows = A.cu_seqlens[b + 1] - t0;
    if (c * kChunk >= rows) return;
    const int tf = t0 + c * kChunk, nt = min(kChunk, rows - c * kChunk);
    const int dk = A.dk, dv = A.dv, H = A.H;
    const int tiles_r = (dk + 63) / 64;
    const int cv0 = (blockIdx.x / tiles_r) * 64, r0 = (blockIdx.x % tiles_r) * 64;
    const int slot = chunk_base(A.cu_seqlens, b) + c;
    // a thread takes sixteen neighbouring tokens of one key row: the products of the decays after each of them, then after their quarter of the chunk
    const int x = threadIdx.x & 63, quarter = threadIdx.x >> 6;
    float k[16], a[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int j = quarter * 16 + i;
        const bool ok = j < nt && r0 + x < dk;
        const int64_t t = tf + (ok ? j : 0);
        k[i] = ok ? A.proj[t * A.ld + A.off_k + h * dk + r0 + x] : 0.f;
        a[i] = ok ? A.alpha[t * A.lda + h * dk + r0 + x] : 1.f;
    }
    for (int e = threadIdx.x; e < kChunk * 64; e += 256) {
        const int j = e >> 6, cx = e & 63;
        vs[j][cx] = (j < nt && cv0 + cx < dv) ? A.proj[(int64_t)(tf + j) * A.ld + A.off_v + h * dv + cv0 + cx] : 0.f;
    }
    float run = 1.f;
#pragma unroll
    for (int i = 15; i >= 0; --i) { k[i] *= run; run *= a[i]; }
    es[quarter][x] = run;
    __syncthreads();
    float tail = 1.f;
    for (int s = quarter + 1; s < 4; ++s) tail *= es[s][x];
#pragma unroll
    for (int i = 0; i < 16; ++i) ks[quarter * 16 + i][x] = k[i] * tail;
    if (quarter == 0 && cv0 == 0 && r0 + x < dk) C.un[((int64_t)slot * H + h) * dk + r0 + x] = run * tail;
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int j = 0; j < nt; ++j) {
        const float4 a4 = *reinterpret_cast<const float4*>(&vs[j][ty * 4]), k4 = *reinterpret_cast<const float4*>(&ks[j][tx * 4]);
        const float va[4] = {a4.x, a4.y, a4.z, a4.w}, ka[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int l = 0; l < 4; ++l) acc[i][l] = fmaf(va[i], ka[l], acc[i][l]);
    }
    float* U = C.U + ((int64_t)slot * H + h) * dv * dk;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int cv = cv0 + ty * 4 + i;
        if (cv >= dv) continue;
#pragma unroll
        for (int l = 0; l < 4; ++l) {
            const int r = r0 + tx * 4 + l;
            if (r < dk) U[(int64_t)cv * dk + r] = acc[i][l];
        }
    }
}

constexpr int kRunPitch = 257;                   // floats per key row of the table of run products: 16 x 16, padded against bank conflicts
constexpr int kChanOutFloats = 3 * 32 * 68 + 2 * 64 * 68 + 32 * 17;

// kBonus: the output is read before the token's own decay and write, so the products of decays leave out the query's token and a token meets its own key and
// value with the bonus weight
template <bool kBonus>
__global__ void __launch_bounds__(256, 2)
la_chan_output_kernel(const ChunkArgs C) {
    pdl_wait();
    pdl_trigger();
    const LinAttnArgs& A = C.A;
    extern __shared__ __align__(16) float sm[];
    float (*qs)[68] = reinterpret_cast<float (*)[68]>(sm);                          // [32][68] q_t P_t of a slab of 32 key rows: [key row][token]
    float (*ks)[68] = reinterpret_cast<float (*)[68]>(sm + 32 * 68);                // [32][68] k_j R_j
    float (*us)[68] = reinterpret_cast<float (*)[68]>(sm + 2 * 32 * 68);            // [32][68] the entering state: [key row][value column]
    float* mm = sm + 3 * 32 * 68;                                                   // [32][257] products of the runs between run b and run a at a * 16 + b (a > b); before run a at a * 17
    float (*pw)[68] = reinterpret_cast<float (*)[68]>(sm + 3 * 32 * 68);            // [64][68] scores: [key token][query token], over the table once the slabs are done
    float (*vs)[68] = reinterpret_cast<float (*)[68]>(sm + 3 * 32 * 68 + 64 * 68);  // [64][68] values: [token][column]
    float* es = sm + 3 * 32 * 68 + 2 * 64 * 68;                                     // [32][17] E of the sixteen runs
    static_assert(32 * kRunPitch <= 2 * 64 * 68, "the table of run products fits under the score and value tiles");
    const int h = blockIdx.y, b = blockIdx.z / C.max_chunks, c = blockIdx.z % C.max_chunks;
    const int t0 = A.cu_seqlens[b], rows = A.cu_seqlens[b + 1] - t0;
    if (c * kChunk >= rows) return;
    const int tf = t0 + c * kChunk, nt = min(kChunk, rows - c * kChunk);
    const int dk = A.dk, dv = A.dv, H = A.H;
    const int cv0 = blockIdx.x * 64;
    const int slot = chunk_base(A.cu_seqlens, b) + c;
    const float* Uin = C.U + ((int64_t)slot * H + h) * dv * dk;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // a thread prepares two runs (warp and warp + 8) of one key row (lane) per slab; the next slab's operands are fetched ahead
    float rq[2][4], rk[2][4], ra[2][4], ru[8], rbo = 0.f;
    auto fetch = [&](int r0) {
        if (kBonus) rbo = r0 + lane < dk ? A.bonus[h * dk + r0 + lane] : 0.f;
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const int j = (warp + 8 * i) * 4 + t;
                const bool ok = j < nt && r0 + lane < dk;
                const int64_t row = tf + (ok ? j : 0);
                rq[i][t] = ok ? A.proj[row * A.ld + A.off_q + h * dk + r0 + lane] * A.q_scale : 0.f;
                rk[i][t] = ok ? A.proj[row * A.ld + A.off_k + h * dk + r0 + lane] : 0.f;
                ra[i][t] = ok ? A.alpha[row * A.lda + h * dk + r0 + lane] : 1.f;
            }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i, j = e >> 5, x = e & 31;
            ru[i] = (cv0 + j < dv && r0 + x < dk) ? Uin[(int64_t)(cv0 + j) * dk + r0 + x] : 0.f;
        }
    };
    float acc[4][4] = {}, o[4][4] = {};
    float dg[2][10] = {};                        // scores inside the thread's two runs: (j, t) for j <= t < 4, this lane's key rows
    fetch(0);
    for (int r0 = 0; r0 < dk; r0 += 32) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int a = warp + 8 * i;
            float p = 1.f, q4[4], k4[4];
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                if (kBonus) q4[t] = rq[i][t] * p;
                p *= ra[i][t];
                if (!kBonus) q4[t] = rq[i][t] * p;
            }
            es[lane * 17 + a] = p;
            float s = 1.f;
#pragma unroll
            for (int t = 3; t >= 0; --t) { k4[t] = rk[i][t] * s; s *= ra[i][t]; }
            *reinterpret_cast<float4*>(&qs[lane][a * 4]) = make_float4(q4[0], q4[1], q4[2], q4[3]);
            *reinterpret_cast<float4*>(&ks[lane][a * 4]) = make_float4(k4[0], k4[1], k4[2], k4[3]);
            int n = 0;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float kj = rk[i][j];
#pragma unroll
                for (int t = j; t < 4; ++t) {
                    if (!kBonus && t > j) kj *= ra[i][t];
                    dg[i][n] = fmaf(rq[i][t], kBonus && t == j ? kj * rbo : kj, dg[i][n]);
                    if (kBonus && t > j) kj *= ra[i][t];
                    ++n;
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int e = threadIdx.x + 256 * i;
            us[e & 31][e >> 5] = ru[i];
        }
        __syncthreads();
        // the table of run products of every key row of the slab: chains of equal total length per warp
        {
            const float* er = es + lane * 17;
            float* mr = mm + lane * kRunPitch;
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int rb = i == 0 ? warp : 15 - warp;
                float m = 1.f;
                for (int a = rb + 1; a < 16; ++a) { mr[a * 16 + rb] = m; m *= er[a]; }
            }
            if (warp == 7) {
                float m = 1.f;
                for (int a = 0; a < 16; ++a) { mr[a * 17] = m; m *= er[a]; }
            }
        }
        __syncthreads();
        if (r0 + 32 < dk) fetch(r0 + 32);
#pragma unroll 4
        for (int x = 0; x < 32; ++x) {
            const float4 q4 = *reinterpret_cast<const float4*>(&qs[x][ty * 4]), k4 = *reinterpret_cast<const float4*>(&ks[x][tx * 4]),
                         u4 = *reinterpret_cast<const float4*>(&us[x][tx * 4]);
            const float m = mm[x * kRunPitch + ty * 16 + tx], before = mm[x * kRunPitch + ty * 17];
            const float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x * m, k4.y * m, k4.z * m, k4.w * m}, u[4] = {u4.x * before, u4.y * before, u4.z * before, u4.w * before};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int l = 0; l < 4; ++l) { acc[i][l] = fmaf(q[i], k[l], acc[i][l]); o[i][l] = fmaf(q[i], u[l], o[i][l]); }
        }
    }
    float rv[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int e = threadIdx.x + 256 * i, j = e >> 6, x = e & 63;
        rv[i] = (j < nt && cv0 + x < dv) ? A.proj[(int64_t)(tf + j) * A.ld + A.off_v + h * dv + cv0 + x] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int n = 0; n < 10; ++n) dg[i][n] = warp_sum(dg[i][n]);
    __syncthreads();                             // the table has been read: its place takes the scores and the values
    if (tx != ty) {                              // an earlier run's keys as summed, a later run's not at all (what was summed there is not a score)
        const bool seen = tx < ty;
#pragma unroll
        for (int l = 0; l < 4; ++l)
            *reinterpret_cast<float4*>(&pw[tx * 4 + l][ty * 4]) = seen ? make_float4(acc[0][l], acc[1][l], acc[2][l], acc[3][l]) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int a = (warp + 8 * i) * 4;
            *reinterpret_cast<float4*>(&pw[a][a]) = make_float4(dg[i][0], dg[i][1], dg[i][2], dg[i][3]);
            *reinterpret_cast<float4*>(&pw[a + 1][a]) = make_float4(0.f, dg[i][4], dg[i][5], dg[i][6]);
            *reinterpret_cast<float4*>(&pw[a + 2][a]) = make_float4(0.f, 0.f, dg[i][7], dg[i][8]);
            *reinterpret_cast<float4*>(&pw[a + 3][a]) = make_float4(0.f, 0.f, 0.f, dg[i][9]);
        }
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int e = threadIdx.x + 256 * i;
        vs[e >> 6][e & 63] = rv[i];
    }
    __syncthreads();
    const int last = min(nt, ty * 4 + 4);        // no key after the thread's last query
#pragma unroll 4
    for (int j = 0; j < last; ++j) {
        const float4 p4 = *reinterpret_cast<const float4*>(&pw[j][ty * 4]), v4 = *reinterpret_cast<const float4*>(&vs[j][tx * 4]);
        const float p[4] = {p4.x, p4.y, p4.z, p4.w}, v[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int l = 0; l < 4; ++l) o[i][l] = fmaf(p[i], v[l], o[i][l]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty * 4 + i;
        if (t >= nt) continue;
#pragma unroll
        for (int l = 0; l < 4; ++l) {
            const int cv = cv0 + tx * 4 + l;
            if (cv < dv) A.out[(int64_t)(tf + t) * H * dv + h * dv + cv] = o[i][l];
        }
    }
}

// ---- every token moved part of the way towards the token before it -------------------------------------------------------------------------------
// out[m, t] = x[t] + (x[t - 1] - x[t]) * mu[m], m = 0 .. mixes - 1, one slab of slab_rows rows per mix; the row before a portion's first comes from
// state [slots, dim] (zero for a new sequence), which then takes the portion's last row: the thread that reads a channel of the state for an entry's first
// row is the one that writes it.  A block walks `rows` rows of kV x 128 channels with the weights and the previous row in registers.
constexpr int kMaxMixes = 8;
template <typename TOut, int kV>
__global__ void __launch_bounds__(128)
token_shift_mix_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ mu, float* __restrict__ state, TOut* __restrict__ out, int64_t slab_rows,
                       const int32_t* __restrict__ token_seq, const int32_t* __restrict__ cu_seqlens, const int32_t* __restrict__ seq_slots,
                       const int32_t* __restrict__ seq_start, int T, int dim, int mixes, int rows) {
    pdl_wait();
    pdl_trigger();
    const int c = (blockIdx.x * 128 + threadIdx.x) * kV;
    if (c >= dim) return;
    const int t_begin = blockIdx.y * rows, t_end = min(T, t_begin + rows);
    auto load = [&](const float* p, float (&v)[kV]) {
        if constexpr (kV == 4) { const float4 f = *reinterpret_cast<const float4*>(p); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
        else v[0] = *p;
    };
    float m[kMaxMixes][kV], prev[kV];
#pragma unroll
    for (int i = 0; i < kMaxMixes; ++i)
        if (i < mixes) load(mu + (int64_t)i * dim + c, m[i]);
    bool have_prev = false;
    for (int t = t_begin; t < t_end; ++t) {
        const int b = token_seq[t], first = cu_seqlens[b];
        float cur[kV];
        load(x + (int64_t)t * ldx + c, cur);
        if (t == first) {
            float* st = state + (int64_t)seq_slots[b] * dim + c;
            if (seq_start[b] == 0) {
#pragma unroll
                for (int j = 0; j < kV; ++j) prev[j] = 0.f;
            } else {
                load(st, prev);
            }
            float last[kV];
            load(x + (int64_t)(cu_seqlens[b + 1] - 1) * ldx + c, last);
#pragma unroll
            for (int j = 0; j < kV; ++j) st[j] = last[j];
        } else if (!have_prev) {
            load(x + (int64_t)(t - 1) * ldx + c, prev);
        }
        have_prev = true;
#pragma unroll
        for (int i = 0; i < kMaxMixes; ++i) {
            if (i >= mixes) break;
            TOut o[kV];
#pragma unroll
            for (int j = 0; j < kV; ++j) o[j] = from_f32<TOut>(fmaf(prev[j] - cur[j], m[i][j], cur[j]));
            TOut* dst = out + ((int64_t)i * slab_rows + t) * dim + c;
            if constexpr (kV == 1) *dst = o[0];
            else if constexpr (sizeof(TOut) == 4) *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(o);
            else *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(o);
        }
#pragma unroll
        for (int j = 0; j < kV; ++j) prev[j] = cur[j];
    }
}

template <int kR, int kG>
void launch_linear_attention(const LinAttnArgs& A, int num_seqs, bool single_rows, cudaStream_t st) {
    if (single_rows) {
        launch_pdl(linear_attention_step_kernel<kR, kG>, dim3(ceil_div(A.dv, 16), A.H, num_seqs), dim3(128), 0, st, A);
        return;
    }
    const int smem = ((kG >= 2 ? 3 : 2) * kTile * 8 * kR + kTile * 16 + 6 * kTile + 1) * (int)sizeof(float);
    ensure_dynamic_smem(reinterpret_cast<const void*>(linear_attention_kernel<kR, kG>), smem);
    launch_pdl(linear_attention_kernel<kR, kG>, dim3(ceil_div(A.dv, 16), A.H, num_seqs), dim3(128), (size_t)smem, st, A);
}

template <int kG>
bool dispatch_linear_attention(const LinAttnArgs& A, int num_seqs, bool single_rows, cudaStream_t st) {
    if (A.dk <= 32) launch_linear_attention<4, kG>(A, num_seqs, single_rows, st);
    else if (A.dk <= 64) launch_linear_attention<8, kG>(A, num_seqs, single_rows, st);
    else if (A.dk <= 128) launch_linear_attention<16, kG>(A, num_seqs, single_rows, st);
    else if (A.dk <= 256) launch_linear_attention<32, kG>(A, num_seqs, single_rows, st);
    else if (A.dk <= 512) launch_linear_attention<64, kG>(A, num_seqs, single_rows, st);      // spills its staging registers: a path for correctness, not speed
    else return false;
    return true;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

void causal_conv_ex(const float* x, int64_t ldx, const float* in_bias, const float* taps, const float* out_bias, float* conv_state, void* y, int64_t ldy,
                    const int32_t* token_seq, const int32_t* cu_seqlens, const int32_t* seq_slots, const int32_t* seq_start, int32_t num_tokens,
                    int32_t num_seqs, int32_t single_rows, int32_t channels, int32_t num_taps, int32_t act, int32_t add_input, int32_t out_dtype, int64_t stream) {
    if (num_tokens == 0 || num_seqs == 0) return;
    B200_REQUIRE(x && taps && conv_state && y && token_seq && cu_seqlens && seq_slots && seq_start && channels > 0 && num_taps >= 1 && ldx >= channels &&
                 ldy >= channels && num_tokens <= 65535 && num_seqs <= 65535 && (act == 0 || act == 1), kErrBadArg, "causal_conv_ex: bad arguments");
    cudaStream_t st = as_stream(stream);
    const dim3 grid(ceil_div(channels, 128), num_tokens);
    if (single_rows) {
        B200_REQUIRE(num_tokens == num_seqs, kErrBadArg, "causal_conv_ex: the single-row kernel takes one row per entry");
        if (out_dtype == B200_F32)
            launch_pdl(causal_conv_step_kernel<float>, grid, dim3(128), 0, st, x, ldx, in_bias, taps, out_bias, conv_state, (float*)y, ldy, seq_slots, seq_start, channels,
                       num_taps, act, add_input);
        else if (out_dtype == B200_BF16)
            launch_pdl(causal_conv_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, x, ldx, in_bias, taps, out_bias, conv_state, (__nv_bfloat16*)y, ldy, seq_slots,
                       seq_start, channels, num_taps, act, add_input);
        else { set_error(kErrUnsupported, "causal_conv_ex: out dtype %d (f32 / bf16)", out_dtype); return; }
        count_launch();
        check_launch("causal_conv_ex");
        return;
    }
    B200_REQUIRE(out_dtype == B200_F32 || out_dtype == B200_BF16, kErrUnsupported, "causal_conv_ex: out dtype %d (f32 / bf16)", out_dtype);
    if (num_tokens > 256 && num_taps <= 8) {
        const bool vec = channels % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && (((uintptr_t)x | (uintptr_t)conv_state | (uintptr_t)y) & 15) == 0;
        const dim3 walk(ceil_div(channels, vec ? 512 : 128), ceil_div(num_tokens, kConvRows));
#define CCW(TO, KK, V) launch_pdl(causal_conv_walk_kernel<TO, KK, V>, walk, dim3(128), 0, st, x, ldx, in_bias, taps, out_bias, (const float*)conv_state, (TO*)y, ldy, token_seq, \
                                  cu_seqlens, seq_slots, seq_start, (int)num_tokens, channels, num_taps, act, add_input)
#define CCW_V(TO, KK) do { if (vec) CCW(TO, KK, 4); else CCW(TO, KK, 1); } while (0)
        if (out_dtype == B200_F32) { if (num_taps <= 4) CCW_V(float, 4); else CCW_V(float, 8); }
        else { if (num_taps <= 4) CCW_V(__nv_bfloat16, 4); else CCW_V(__nv_bfloat16, 8); }
#undef CCW_V
#undef CCW
    } else if (out_dtype == B200_F32)
        launch_pdl(causal_conv_ex_kernel<float>, grid, dim3(128), 0, st, x, ldx, in_bias, taps, out_bias, (const float*)conv_state, (float*)y, ldy, token_seq,
                   cu_seqlens, seq_slots, seq_start, channels, num_taps, act, add_input);
    else
        launch_pdl(causal_conv_ex_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, x, ldx, in_bias, taps, out_bias, (const float*)conv_state, (__nv_bfloat16*)y, ldy,
                   token_seq, cu_seqlens, seq_slots, seq_start, channels, num_taps, act, add_input);
    count_launch();
    if (num_taps > 1) {
        launch_pdl(causal_conv_roll_kernel, dim3(ceil_div(channels, 128), num_seqs), dim3(128), 0, st, x, ldx, in_bias, conv_state, cu_seqlens, seq_slots, seq_start,
                   channels, num_taps);
        count_launch();
    }
    check_launch("causal_conv_ex");
}

void block_diag_linear(const float* x, int64_t ldx, const float* weight, const float* bias, float* out, int64_t ldy, int32_t num_tokens, int32_t blocks,
                       int32_t rows_per_block, int32_t cols_per_block, int64_t stream) {
    if (num_tokens == 0) return;
    B200_REQUIRE(x && weight && out && blocks > 0 && blocks <= 65535 && rows_per_block > 0 && cols_per_block > 0 && ldx >= (int64_t)blocks * cols_per_block &&
                 ldy >= (int64_t)blocks * rows_per_block, kErrBadArg, "block_diag_linear: bad arguments");
    cudaStream_t st = as_stream(stream);
    if (num_tokens <= 8)
        launch_pdl(block_diag_rows_kernel, dim3(ceil_div(rows_per_block, 8), ceil_div(num_tokens, 4), blocks), dim3(256), 0, st, x, ldx, weight, bias, out, ldy,
                   num_tokens, rows_per_block, cols_per_block);
    else
        launch_pdl(block_diag_linear_kernel, dim3(ceil_div(rows_per_block, kBN), ceil_div(num_tokens, kBM), blocks), dim3(256), 0, st, x, ldx, weight, bias, out, ldy,
                   num_tokens, rows_per_block, cols_per_block);
    count_launch();
    check_launch("block_diag_linear");
}

void gated_linear_scan(const float* u, int64_t ldu, float* gates, int64_t ld_gates, const float* lam, float* y_pre, int64_t ldy, const float* y_bias,
                       float* state, void* out, float* scratch, const int32_t* cu_seqlens, const int32_t* seq_slots, const int32_t* seq_start, int32_t num_tokens, int32_t num_seqs,
                       int32_t max_rows, int32_t channels, int32_t block_channels, float decay_scale, int32_t out_dtype, int64_t stream) {
    if (num_seqs == 0 || num_tokens == 0) return;
    B200_REQUIRE(u && gates && lam && y_pre && state && out && cu_seqlens && seq_slots && seq_start && channels > 0 && block_channels > 0 &&
                 channels % block_channels == 0 && ldu >= channels && ldy >= channels && ld_gates >= 2 * (int64_t)channels && num_seqs <= 65535, kErrBadArg,
                 "gated_linear_scan: bad arguments");
    B200_REQUIRE(out_dtype == B200_F32 || out_dtype == B200_BF16, kErrUnsupported, "gated_linear_scan: out dtype %d (f32 / bf16)", out_dtype);
    cudaStream_t st = as_stream(stream);
    if (max_rows >= kScanSplitRows) {
        // portions of prompts: everything but the recurrence itself for all rows at once (in place), then a scan of two multiply-adds per row
        const int64_t total = (int64_t)num_tokens * channels;
        launch_pdl(gated_scan_prepare_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st, u, ldu, gates, ld_gates, lam, y_pre, ldy, y_bias,
                   (int64_t)num_tokens, channels, block_channels, decay_scale);
        if (max_rows >= kScanChunkedRows && scratch && (int64_t)ceil_div(max_rows, kScanChunk) * num_seqs <= 65535) {
            const int max_chunks = ceil_div(max_rows, kScanChunk);
            const dim3 cgrid(ceil_div(channels, 128), max_chunks, num_seqs);
            launch_pdl(scan_chunk_compose_kernel, cgrid, dim3(128), 0, st, (const float*)gates, ld_gates, scratch, cu_seqlens, channels, block_channels);
            launch_pdl(scan_chunk_carry_kernel, dim3(ceil_div(channels, 128), num_seqs), dim3(128), 0, st, scratch, state, cu_seqlens, seq_slots, seq_start, channels);
            if (out_dtype == B200_F32)
                launch_pdl(scan_chunk_replay_kernel<float>, cgrid, dim3(128), 0, st, (const float*)gates, ld_gates, (const float*)y_pre, ldy, (const float*)scratch,
                           (float*)out, cu_seqlens, channels, block_channels);
            else
                launch_pdl(scan_chunk_replay_kernel<__nv_bfloat16>, cgrid, dim3(128), 0, st, (const float*)gates, ld_gates, (const float*)y_pre, ldy,
                           (const float*)scratch, (__nv_bfloat16*)out, cu_seqlens, channels, block_channels);
            count_launch(4);
            check_launch("gated_linear_scan");
            return;
        }
        const dim3 grid(ceil_div(channels, 32), num_seqs);
        if (out_dtype == B200_F32)
            launch_pdl(linear_scan_kernel<float>, grid, dim3(32), 0, st, (const float*)gates, ld_gates, (const float*)y_pre, ldy, state, (float*)out, cu_seqlens, seq_slots,
                       seq_start, channels, block_channels);
        else
            launch_pdl(linear_scan_kernel<__nv_bfloat16>, grid, dim3(32), 0, st, (const float*)gates, ld_gates, (const float*)y_pre, ldy, state, (__nv_bfloat16*)out,
                       cu_seqlens, seq_slots, seq_start, channels, block_channels);
        count_launch(2);
        check_launch("gated_linear_scan");
        return;
    }
    const dim3 grid(ceil_div(channels, 64), num_seqs);
    if (out_dtype == B200_F32)
        launch_pdl(gated_linear_scan_kernel<float>, grid, dim3(64), 0, st, u, ldu, (const float*)gates, ld_gates, lam, (const float*)y_pre, ldy, y_bias, state, (float*)out,
                   cu_seqlens, seq_slots, seq_start, channels, block_channels, decay_scale);
    else
        launch_pdl(gated_linear_scan_kernel<__nv_bfloat16>, grid, dim3(64), 0, st, u, ldu, (const float*)gates, ld_gates, lam, (const float*)y_pre, ldy, y_bias, state,
                   (__nv_bfloat16*)out, cu_seqlens, seq_slots, seq_start, channels, block_channels, decay_scale);
    count_launch();
    check_launch("gated_linear_scan");
}

void linear_attention(const float* proj, int64_t ld, int32_t off_q, int32_t off_k, int32_t off_v, int32_t off_i, int32_t off_f, const float* decay,
                      const float* i_bias, const float* f_bias, float gate_cap, float q_scale, int32_t act, int32_t gating, float* state, float* normaliser,
                      float* maximum, float* out, const int32_t* cu_seqlens, const int32_t* seq_slots, const int32_t* seq_start, int32_t num_tokens,
                      int32_t num_seqs, int32_t single_rows, int32_t num_heads, int32_t dk, int32_t dv, int64_t stream) {
    if (num_seqs == 0) return;
    B200_REQUIRE(!single_rows || num_tokens == num_seqs, kErrBadArg, "linear_attention: the single-row kernel takes one row per entry");
    B200_REQUIRE(proj && state && out && cu_seqlens && seq_slots && seq_start && num_heads > 0 && num_heads <= 65535 && num_seqs <= 65535 && dk > 0 && dv > 0 &&
                 (act == 0 || act == 1) && (gating == 0 || gating == 1), kErrBadArg, "linear_attention: bad arguments");
    B200_REQUIRE(gating == 0 ? decay != nullptr : (normaliser && maximum && gate_cap > 0.f), kErrBadArg,
                 "linear_attention: fixed decay needs decay[H]; exponential gating needs the normaliser, the maximum and a positive cap");
    B200_REQUIRE(dk <= 512, kErrUnsupported, "linear_attention: key size %d > 512", dk);
    LinAttnArgs A{proj, ld, off_q, off_k, off_v, off_i, off_f, decay, i_bias, f_bias, gate_cap, q_scale, act, state, normaliser, maximum, out,
                  cu_seqlens, seq_slots, seq_start, num_heads, dk, dv, nullptr, 0, nullptr};
    cudaStream_t st = as_stream(stream);
    if (gating == 0) dispatch_linear_attention<0>(A, num_seqs, single_rows != 0, st);
    else dispatch_linear_attention<1>(A, num_seqs, single_rows != 0, st);
    count_launch();
    check_launch("linear_attention");
}

int64_t linear_attention_chunked_scratch(int32_t num_tokens, int32_t num_seqs, int32_t num_heads, int32_t dk, int32_t dv) {
    // floats: per chunk slot a [dv, dk] term per head and two normaliser rows, per token three gate values per head, per entry a maximum per head
    const int64_t slots = (int64_t)(num_tokens + kChunk - 1) / kChunk + num_seqs;
    return slots * num_heads * ((int64_t)dv * dk + 2 * dk) + (int64_t)num_tokens * num_heads * 3 + (int64_t)num_seqs * num_heads;
}


void linear_attention_chunked(const float* proj, int64_t ld, int32_t off_q, int32_t off_k, int32_t off_v, int32_t off_i, int32_t off_f, const float* decay,
                              const float* i_bias, const float* f_bias, float gate_cap, float q_scale, int32_t act, int32_t gating, float* state, float* normaliser,
                              float* maximum, float* out, float* scratch, const int32_t* cu_seqlens, const int32_t* seq_slots, const int32_t* seq_start,
                              int32_t num_tokens, int32_t num_seqs, int32_t max_rows, int32_t num_heads, int32_t dk, int32_t dv, int64_t stream) {
    if (num_seqs == 0 || num_tokens == 0) return;
    B200_REQUIRE(proj && state && out && scratch && cu_seqlens && seq_slots && seq_start && num_heads > 0 && num_heads <= 65535 && dk > 0 && dv > 0 && max_rows > 0 &&
                 (act == 0 || act == 1) && (gating == 0 || gating == 1), kErrBadArg, "linear_attention_chunked: bad arguments");
    B200_REQUIRE(gating == 0 ? decay != nullptr : (normaliser && maximum && gate_cap > 0.f), kErrBadArg,
                 "linear_attention_chunked: fixed decay needs decay[H]; exponential gating needs the normaliser, the maximum and a positive cap");
    const int max_chunks = (max_rows + kChunk - 1) / kChunk;
    B200_REQUIRE((int64_t)max_chunks * num_seqs <= 65535, kErrUnsupported, "linear_attention_chunked: %d chunks x %d entries exceed the grid", max_chunks, num_seqs);
    const int64_t slots = (int64_t)(num_tokens + kChunk - 1) / kChunk + num_seqs;
    ChunkArgs C;
    C.A = LinAttnArgs{proj, ld, off_q, off_k, off_v, off_i, off_f, decay, i_bias, f_bias, gate_cap, q_scale, act, state, normaliser, maximum, out,
                      cu_seqlens, seq_slots, seq_start, num_heads, dk, dv, nullptr, 0, nullptr};
    C.U = scratch;
    C.un = C.U + slots * num_heads * dv * dk;
    C.un_in = C.un + slots * num_heads * dk;
    C.gc = C.un_in + slots * num_heads * dk;
    C.m0 = C.gc + (int64_t)num_tokens * num_heads * 3;
    C.max_chunks = max_chunks;
    C.gating = gating;
    cudaStream_t st = as_stream(stream);
    int launches = 3;
    if (gating == 1) {
        launch_pdl(la_gate_values_kernel, dim3(ceil_div((int64_t)num_tokens * num_heads, 256)), dim3(256), 0, st, C, (int)num_tokens);
        launch_pdl(la_gate_chain_kernel, dim3(ceil_div(num_heads, 32), num_seqs), dim3(32), 0, st, C);
        launches += 2;
    }
    const unsigned z = (unsigned)(max_chunks * num_seqs);
    launch_pdl(la_chunk_state_kernel, dim3(ceil_div(dv, 64) * ceil_div(dk, 64), num_heads, z), dim3(256), 0, st, C);
    launch_pdl(la_chunk_scan_kernel, dim3(ceil_div((int64_t)num_heads * dv * dk, 256), num_seqs), dim3(256), 0, st, C);
    const int smem = (2 * 32 * 68 + 2 * 64 * 68 + 5 * 64) * (int)sizeof(float);
    ensure_dynamic_smem(reinterpret_cast<const void*>(la_chunk_output_kernel), smem);
    launch_pdl(la_chunk_output_kernel, dim3(ceil_div(dv, 64), num_heads, z), dim3(256), (size_t)smem, st, C);
    count_launch(launches);
    check_launch("linear_attention_chunked");
}

void low_rank_decay(const float* y, int64_t ldy, const float* weight, const float* bias, float* alpha, int32_t num_tokens, int32_t channels, int32_t rank, float tau,
                    int64_t stream) {
    low_rank_map(y, ldy, weight, bias, alpha, num_tokens, channels, rank, 0, 0, tau, nullptr, 1, stream);
}

void low_rank_map(const float* y, int64_t ldy, const float* weight, const float* bias, float* out, int32_t num_tokens, int32_t channels, int32_t rank, int32_t in_tanh,
                  int32_t form, float tau, const float* log_rate, int32_t channels_per_rate, int64_t stream) {
    if (num_tokens == 0) return;
    B200_REQUIRE(y && weight && out && channels > 0 && rank > 0 && ldy >= rank && num_tokens <= 32 * 65535 && form >= 0 && form <= 3 && (form != 0 || tau > 0.f) &&
                 (form != 2 || (log_rate && channels_per_rate > 0 && channels % channels_per_rate == 0)), kErrBadArg, "low_rank_map: bad arguments");
    cudaStream_t st = as_stream(stream);
    const float inv_tau = form == 0 ? 1.0f / tau : 0.f;
    if (num_tokens <= 256)
        launch_pdl(low_rank_rows_kernel, dim3(ceil_div(channels, 32), ceil_div(num_tokens, 32)), dim3(256), 0, st, y, ldy, weight, bias, out, (int)num_tokens, (int)channels,
                   (int)rank, inv_tau, (int)in_tanh, (int)form, log_rate, (int)channels_per_rate);
    else
        launch_pdl(low_rank_tile_kernel, dim3(ceil_div(channels, 128), ceil_div(num_tokens, 64)), dim3(256), 0, st, y, ldy, weight, bias, out, (int)num_tokens, (int)channels,
                   (int)rank, inv_tau, (int)in_tanh, (int)form, log_rate, (int)channels_per_rate);
    count_launch();
    check_launch("low_rank_map");
}

void token_shift_mix(const float* x, int64_t ldx, const float* mu, float* state, void* out, int64_t slab_rows, const int32_t* token_seq, const int32_t* cu_seqlens,
                     const int32_t* seq_slots, const int32_t* seq_start, int32_t num_tokens, int32_t dim, int32_t mixes, int32_t out_dtype, int64_t stream) {
    if (num_tokens == 0) return;
    B200_REQUIRE(x && mu && state && out && token_seq && cu_seqlens && seq_slots && seq_start && dim > 0 && ldx >= dim && slab_rows >= num_tokens && mixes >= 1 && mixes <= kMaxMixes,
                 kErrBadArg, "token_shift_mix: bad arguments (1 to %d mixes)", kMaxMixes);
    B200_REQUIRE(out_dtype == B200_F32 || out_dtype == B200_BF16, kErrUnsupported, "token_shift_mix: out dtype %d (f32 / bf16)", out_dtype);
    const bool vec = dim % 4 == 0 && ldx % 4 == 0 && (((uintptr_t)x | (uintptr_t)mu | (uintptr_t)state | (uintptr_t)out) & 15) == 0;
    const int rows = num_tokens <= 256 ? 1 : 8;
    const dim3 grid(ceil_div(dim, vec ? 512 : 128), ceil_div(num_tokens, rows));
    cudaStream_t st = as_stream(stream);
#define TSM(TO, V) launch_pdl(token_shift_mix_kernel<TO, V>, grid, dim3(128), 0, st, x, ldx, mu, state, (TO*)out, slab_rows, token_seq, cu_seqlens, seq_slots, seq_start, \
                              (int)num_tokens, (int)dim, (int)mixes, rows)
    if (out_dtype == B200_F32) { if (vec) TSM(float, 4); else TSM(float, 1); }
    else { if (vec) TSM(__nv_bfloat16, 4); else TSM(__nv_bfloat16, 1); }
#undef TSM
    count_launch();
    check_launch("token_shift_mix");
}

void linear_attention_channel(const float* proj, int64_t ld, int32_t off_q, int32_t off_k, int32_t off_v, const float* alpha, int64_t lda, float q_scale, float* state,
                              float* out, float* scratch, const int32_t* cu_seqlens, const int32_t* seq_slots, const int32_t* seq_start, int32_t num_tokens,
                              int32_t num_seqs, int32_t max_rows, int32_t mode, int32_t num_heads, int32_t dk, int32_t dv, int64_t stream) {
    linear_attention_channel_bonus(proj, ld, off_q, off_k, off_v, alpha, lda, nullptr, q_scale, state, out, scratch, cu_seqlens, seq_slots, seq_start, num_tokens, num_seqs,
                                   max_rows, mode, num_heads, dk, dv, stream);
}

void linear_attention_channel_bonus(const float* proj, int64_t ld, int64_t off_q, int64_t off_k, int64_t off_v, const float* alpha, int64_t lda, const float* bonus,
                                    float q_scale, float* state, float* out, float* scratch, const int32_t* cu_seqlens, const int32_t* seq_slots,
                                    const int32_t* seq_start, int32_t num_tokens, int32_t num_seqs, int32_t max_rows, int32_t mode, int32_t num_heads, int32_t dk,
                                    int32_t dv, int64_t stream) {
    if (num_seqs == 0 || num_tokens == 0) return;
    B200_REQUIRE(proj && alpha && state && out && cu_seqlens && seq_slots && seq_start && num_heads > 0 && num_heads <= 65535 && num_seqs <= 65535 && dk > 0 && dv > 0 &&
                 lda >= (int64_t)num_heads * dk && mode >= 0 && mode <= 2, kErrBadArg, "linear_attention_channel: bad arguments");
    // the three operands may be columns of one matrix or matrices of their own with one pitch: an offset is anything from the first to the last element
    LinAttnArgs A{proj, ld, off_q, off_k, off_v, 0, 0, nullptr, nullptr, nullptr, 0.f, q_scale, 0, state, nullptr, nullptr, out,
                  cu_seqlens, seq_slots, seq_start, num_heads, dk, dv, alpha, lda, bonus};
    cudaStream_t st = as_stream(stream);
    if (mode != 2) {
        B200_REQUIRE(mode == 0 || num_tokens == num_seqs, kErrBadArg, "linear_attention_channel: the single-row kernel takes one row per entry");
        B200_REQUIRE(dk <= 512, kErrUnsupported, "linear_attention_channel: key size %d > 512", dk);
        if (bonus) dispatch_linear_attention<3>(A, num_seqs, mode == 1, st);
        else dispatch_linear_attention<2>(A, num_seqs, mode == 1, st);
        count_launch();
        check_launch("linear_attention_channel");
        return;
    }
    B200_REQUIRE(scratch && max_rows > 0, kErrBadArg, "linear_attention_channel: the chunked form needs scratch and max_rows");
    const int max_chunks = (max_rows + kChunk - 1) / kChunk;
    B200_REQUIRE((int64_t)max_chunks * num_seqs <= 65535, kErrUnsupported, "linear_attention_channel: %d chunks x %d entries exceed the grid", max_chunks, num_seqs);
    const int64_t slots = (int64_t)(num_tokens + kChunk - 1) / kChunk + num_seqs;
    ChunkArgs C{};
    C.A = A;
    C.U = scratch;
    C.un = C.U + slots * num_heads * dv * dk;
    C.max_chunks = max_chunks;
    C.gating = 2;
    const unsigned z = (unsigned)(max_chunks * num_seqs);
    launch_pdl(la_chan_state_kernel, dim3(ceil_div(dv, 64) * ceil_div(dk, 64), num_heads, z), dim3(256), 0, st, C);
    launch_pdl(la_chunk_scan_kernel, dim3(ceil_div((int64_t)num_heads * dv * dk, 256), num_seqs), dim3(256), 0, st, C);
    const int smem = kChanOutFloats * (int)sizeof(float);
    void (*output)(const ChunkArgs) = bonus ? la_chan_output_kernel<true> : la_chan_output_kernel<false>;
    ensure_dynamic_smem(reinterpret_cast<const void*>(output), smem);
    launch_pdl(output, dim3(ceil_div(dv, 64), num_heads, z), dim3(256), (size_t)smem, st, C);
    count_launch(3);
    check_launch("linear_attention_channel");
}

}  // extern "C"
