// delta_chunk.cu -- the gated delta rule with a decay per token and key row over chunks of 64 tokens, for portions of prompts; all arithmetic f32.
//
// Per head, with S [dk, dv]:  S <- diag(g_t) S;  u_t = beta_t (v_t - S^T k_t);  S <- S + k_t u_t^T;  o_t = S^T q_t.  Inside a chunk that is entered with the state S0,
// with P_t = g_0 ... g_t and R_ts = g_(s+1) ... g_t per key row,
//     u_t = beta_t (v_t - (P_t k_t)^T S0 - sum_{s<t} M_ts u_s),      M_ts = sum_r k_t[r] R_ts[r] k_s[r]
//     o_t = (P_t q_t)^T S0 + sum_{s<=t} N_ts u_s,                    N_ts = sum_r q_t[r] R_ts[r] k_s[r]
//     S_end = diag(P_last) S0 + sum_s (R_last,s k_s) u_s^T
// The triangular system does not involve the state: with B = (I + diag(beta) strict(M))^-1 diag(beta), U = B V - (B K_P) S0, where K_P holds the rows P_t k_t.  B's entries are
// responses of the recurrence itself, which contracts (beta <= 1, unit keys, decays <= 1), so they stay of order one.  Three kernels:
//   delta_chunk_prepare  per (chunk, head), all at once: unit vectors, decay products, M, N, B, W = B K_P, U0 = B V, the rows P_t q_t and R_last,s k_s
//   delta_chunk_walk     per (entry, head, 16 value columns) the walk over the chunks: U = U0 - W S0, then S_end; leaves U and the state entering every chunk
//   delta_chunk_output   per (chunk, head, 64 or 128 value columns), all at once: o
// Decays enter as products only, each in [0, 1]: tokens in runs of four, prefix and suffix products inside a run, a table per key row of the products of whole runs
// between two runs.  Nothing overflows, and a product that underflows is a contribution that has died.
#include "common.cuh"

namespace b200 {
namespace {

constexpr int kC = 64;                           // tokens per chunk
constexpr int kLd = 68;                          // row pitch of 64-wide tiles: 16-byte reads of neighbours, rows four banks apart
constexpr int kRunPitch = 273;                   // per key row: products of the runs between two runs (16 x 16), before a run (diagonal), after a run (256 + run)

struct DeltaChunkArgs {
    const float* qkv; const float* proj; int64_t ld_proj; int off_b;
    const float* decay;                          // [T, H dk]
    float* state; float* out;                    // [slots, H, dv, dk], [T, H dv]
    const int32_t* cu; const int32_t* slots; const int32_t* start;
    int T, H, G, dk, dv, max_chunks;
    float *W, *KE;                               // [T, H, dk]
    float* QP;                                   // [chunks, H, dk, 64]: tokens innermost, the layout the output kernel multiplies from
    float* N;                                    // [chunks, H, 64 (s), 64 (t)]
    float* U;                                    // [T, H, dv]
    float* Pe;                                   // [chunks, H, dk] the product of a chunk's decays
    float* Sc;                                   // [chunks, H, dk, dv] the state entering a chunk
};

__host__ __device__ __forceinline__ int64_t chunk_slots(int T, int B) { return (T + kC - 1) / kC + B; }
__device__ __forceinline__ int chunk_base(const int32_t* cu, int b) {      // chunks of the entries before b
    int s = 0;
    for (int i = 0; i < b; ++i) s += (cu[i + 1] - cu[i] + kC - 1) / kC;
    return s;
}

__device__ __forceinline__ void cp_async(float* dst, const float* src, bool ok, bool wide) {       // 16 or 4 bytes; zeros where the source does not exist
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if (wide) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(ok ? 16 : 0) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(ok ? 4 : 0) : "memory");
}

constexpr int kPrepFloats(int kd) { return 3 * 32 * kLd + 32 * kRunPitch + 32 * 17 + kC * (kd + 4) + 3 * kC; }

template <int kKD>
__global__ void __launch_bounds__(256, 2)
delta_chunk_prepare_kernel(const DeltaChunkArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr int kKp = kKD + 4;
    extern __shared__ __align__(16) float sm[];
    float (*qs)[kLd] = reinterpret_cast<float (*)[kLd]>(sm);                        // [32][68] q times its own run's prefix: [key row][token]
    float (*ka)[kLd] = reinterpret_cast<float (*)[kLd]>(sm + 32 * kLd);             // [32][68] k times its own run's prefix
    float (*kb)[kLd] = reinterpret_cast<float (*)[kLd]>(sm + 2 * 32 * kLd);         // [32][68] k times its own run's suffix
    float* mm = sm + 3 * 32 * kLd;                                                  // [32][273] products of runs
    float* es = mm + 32 * kRunPitch;                                                // [32][17] product of each run
    float* KP = es + 32 * 17;                                                       // [64][kKp] P_t k_t
    float* qn = KP + kC * kKp;                                                      // [64] norms, then beta
    float* kn = qn + kC;
    float* bs = kn + kC;
    float (*Mt)[kLd] = reinterpret_cast<float (*)[kLd]>(mm);                        // [s][t], over the table once the slabs are done
    float (*Bt)[kLd] = reinterpret_cast<float (*)[kLd]>(mm + kC * kLd);             // [s][t]
    float (*Vs)[kLd] = reinterpret_cast<float (*)[kLd]>(sm);                        // [s][column], over the slabs
    static_assert(2 * kC * kLd <= 32 * kRunPitch && kC * kLd <= 3 * 32 * kLd, "tiles fit over the tables they replace");
    const int h = blockIdx.y, b = blockIdx.z / A.max_chunks, c = blockIdx.z % A.max_chunks;
    const int t0 = A.cu[b], rows = A.cu[b + 1] - t0;
    if (c * kC >= rows) return;
    const int tf = t0 + c * kC, nt = min(kC, rows - c * kC);
    const int dk = A.dk, dv = A.dv, H = A.H, g = h / (H / A.G);
    const int64_t ch = (int64_t)(chunk_base(A.cu, b) + c) * H + h;
    float* QPt = A.QP + ch * dk * kC;
    float* Nt = A.N + ch * kC * kC;
    const int C = 2 * A.G * dk + H * dv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const float* qbase = A.qkv + (int64_t)tf * C + g * dk;
    const float* kbase = qbase + A.G * dk;
#pragma unroll 4
    for (int i = 0; i < kC / 8; ++i) {
        const int t = warp + 8 * i;
        float qq = 0.f, kk = 0.f;
#pragma unroll
        for (int r4 = 0; r4 < kKD / 32; ++r4) {
            const int r = lane + 32 * r4;
            const bool ok = t < nt && r < dk;
            const float x = ok ? qbase[(int64_t)t * C + r] : 0.f, y = ok ? kbase[(int64_t)t * C + r] : 0.f;
            qq = fmaf(x, x, qq); kk = fmaf(y, y, kk);
        }
        qq = warp_sum(qq); kk = warp_sum(kk);
        if (lane == 0) {
            qn[t] = (1.0f / sqrtf((float)dk)) / sqrtf(qq + 1e-6f);
            kn[t] = 1.0f / sqrtf(kk + 1e-6f);
            bs[t] = t < nt ? 1.0f / (1.0f + expf(-A.proj[(int64_t)(tf + t) * A.ld_proj + A.off_b + h])) : 0.f;
        }
    }
    __syncthreads();
    // ---- the two score matrices, a slab of 32 key rows at a time; a thread prepares two runs (warp and warp + 8) of one key row (lane) ------------------
    float rq[2][4], rk[2][4], ra[2][4];
    auto fetch = [&](int r0) {
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const int j = (warp + 8 * i) * 4 + t;
                const bool ok = j < nt && r0 + lane < dk;
                rq[i][t] = ok ? qbase[(int64_t)j * C + r0 + lane] * qn[j] : 0.f;
                rk[i][t] = ok ? kbase[(int64_t)j * C + r0 + lane] * kn[j] : 0.f;
                ra[i][t] = ok ? A.decay[(int64_t)(tf + j) * H * dk + h * dk + r0 + lane] : 1.f;
            }
    };
    // the 120 tiles (run of queries, earlier run of keys) below the diagonal go to threads 0 .. 239 in pairs: an even thread takes N's tile, an odd one M's
    int tq = 1;
    while (tq * (tq + 1) / 2 <= (int)(threadIdx.x >> 1) && tq < 15) ++tq;
    const int tk = min((int)(threadIdx.x >> 1) - tq * (tq - 1) / 2, 15);
    const bool has_tile = threadIdx.x < 240;
    float as[4][4] = {};
    float dn[2][10] = {}, dm[2][6] = {};         // inside the thread's two runs, this lane's key rows: N for s <= t, M for s < t
    fetch(0);
    for (int r0 = 0; r0 < dk; r0 += 32) {
        float a4[2][4], b4[2][4];
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int a = warp + 8 * i;
            float p = 1.f, s = 1.f, q4[4];
#pragma unroll
            for (int t = 0; t < 4; ++t) { p *= ra[i][t]; q4[t] = rq[i][t] * p; a4[i][t] = rk[i][t] * p; }
#pragma unroll
            for (int t = 3; t >= 0; --t) { b4[i][t] = rk[i][t] * s; s *= ra[i][t]; }
            es[lane * 17 + a] = p;
            *reinterpret_cast<float4*>(&qs[lane][a * 4]) = make_float4(q4[0], q4[1], q4[2], q4[3]);
            *reinterpret_cast<float4*>(&ka[lane][a * 4]) = make_float4(a4[i][0], a4[i][1], a4[i][2], a4[i][3]);
            *reinterpret_cast<float4*>(&kb[lane][a * 4]) = make_float4(b4[i][0], b4[i][1], b4[i][2], b4[i][3]);
            int n = 0, m = 0;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float kj = rk[i][j];
#pragma unroll
                for (int t = j; t < 4; ++t) {
                    if (t > j) { kj *= ra[i][t]; dm[i][m] = fmaf(rk[i][t], kj, dm[i][m]); ++m; }
                    dn[i][n] = fmaf(rq[i][t], kj, dn[i][n]);
                    ++n;
                }
            }
        }
        __syncthreads();
        {
            const float* er = es + lane * 17;
            float* mr = mm + lane * kRunPitch;
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int rb = i == 0 ? warp : 15 - warp;
                float m = 1.f;
                for (int a = rb + 1; a < 16; ++a) { mr[a * 16 + rb] = m; m *= er[a]; }
                mr[256 + rb] = m;                              // the runs after run rb
            }
            if (warp == 7) {
                float m = 1.f;
                for (int a = 0; a < 16; ++a) { mr[a * 17] = m; m *= er[a]; }
                if (r0 + lane < dk) A.Pe[ch * dk + r0 + lane] = m;
            }
        }
        __syncthreads();
        if (r0 + lane < dk) {
            const float* mr = mm + lane * kRunPitch;
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int a = warp + 8 * i;
                const float before = mr[a * 17], after = mr[256 + a];
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    const int j = a * 4 + t;
                    KP[j * kKp + r0 + lane] = a4[i][t] * before;
                    if (j >= nt) continue;
                    A.KE[((int64_t)(tf + j) * H + h) * dk + r0 + lane] = b4[i][t] * after;
                }
            }
        } else if (r0 + lane < kKp) {
#pragma unroll
            for (int i = 0; i < 8; ++i) KP[((warp + 8 * (i >> 2)) * 4 + (i & 3)) * kKp + r0 + lane] = 0.f;
        }
        if (r0 + 32 < dk) fetch(r0 + 32);
#pragma unroll
        for (int i = 0; i < 2; ++i) {                          // P_t q_t, a run of four tokens at a time
            const int x = (threadIdx.x >> 4) + 16 * i;
            if (r0 + x >= dk) continue;
            const float before = mm[x * kRunPitch + tx * 17];
            const float4 q = *reinterpret_cast<const float4*>(&qs[x][tx * 4]);
            *reinterpret_cast<float4*>(QPt + (int64_t)(r0 + x) * kC + tx * 4) = make_float4(q.x * before, q.y * before, q.z * before, q.w * before);
        }
        if (has_tile) {
            const float* left = (threadIdx.x & 1) ? &ka[0][tq * 4] : &qs[0][tq * 4];
            const float* right = &kb[0][tk * 4];
            const float* mid = mm + tq * 16 + tk;
#pragma unroll 8
            for (int x = 0; x < 32; ++x) {
                const float m = mid[x * kRunPitch];
                const float4 q = *reinterpret_cast<const float4*>(left + x * kLd), e = *reinterpret_cast<const float4*>(right + x * kLd);
                const float qv[4] = {q.x, q.y, q.z, q.w}, ev[4] = {e.x * m, e.y * m, e.z * m, e.w * m};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int l = 0; l < 4; ++l) as[i][l] = fmaf(qv[i], ev[l], as[i][l]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
#pragma unroll
        for (int n = 0; n < 10; ++n) dn[i][n] = warp_sum(dn[i][n]);
#pragma unroll
        for (int n = 0; n < 6; ++n) dm[i][n] = warp_sum(dm[i][n]);
    }
    __syncthreads();                                           // the table has been read: its place takes M and B
    // tiles on the diagonal are filled by their runs' owners below, scores over later tokens are zero
    if (has_tile) {
#pragma unroll
        for (int l = 0; l < 4; ++l) {
            const float4 v = make_float4(as[0][l], as[1][l], as[2][l], as[3][l]);
            if (threadIdx.x & 1) *reinterpret_cast<float4*>(&Mt[tk * 4 + l][tq * 4]) = v;
            else *reinterpret_cast<float4*>(Nt + (tk * 4 + l) * kC + tq * 4) = v;
        }
    }
    if (tx > ty) {
#pragma unroll
        for (int l = 0; l < 4; ++l) {
            *reinterpret_cast<float4*>(&Mt[tx * 4 + l][ty * 4]) = make_float4(0.f, 0.f, 0.f, 0.f);
            *reinterpret_cast<float4*>(Nt + (tx * 4 + l) * kC + ty * 4) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int a = (warp + 8 * i) * 4;
            *reinterpret_cast<float4*>(&Mt[a][a]) = make_float4(0.f, dm[i][0], dm[i][1], dm[i][2]);
            *reinterpret_cast<float4*>(&Mt[a + 1][a]) = make_float4(0.f, 0.f, dm[i][3], dm[i][4]);
            *reinterpret_cast<float4*>(&Mt[a + 2][a]) = make_float4(0.f, 0.f, 0.f, dm[i][5]);
            *reinterpret_cast<float4*>(&Mt[a + 3][a]) = make_float4(0.f, 0.f, 0.f, 0.f);
            *reinterpret_cast<float4*>(Nt + a * kC + a) = make_float4(dn[i][0], dn[i][1], dn[i][2], dn[i][3]);
            *reinterpret_cast<float4*>(Nt + (a + 1) * kC + a) = make_float4(0.f, dn[i][4], dn[i][5], dn[i][6]);
            *reinterpret_cast<float4*>(Nt + (a + 2) * kC + a) = make_float4(0.f, 0.f, dn[i][7], dn[i][8]);
            *reinterpret_cast<float4*>(Nt + (a + 3) * kC + a) = make_float4(0.f, 0.f, 0.f, dn[i][9]);
        }
    }
    // the first 64 value columns travel while B is worked out
    const float* vrow = A.qkv + (int64_t)tf * C + 2 * A.G * dk + h * dv;
    const bool wide_v = (dv & 3) == 0 && (C & 3) == 0 && ((2 * A.G * dk) & 3) == 0 && ((uintptr_t)A.qkv & 15) == 0;
    auto issue_values = [&](int c0) {
        const int w = wide_v ? 4 : 1;
        for (int e = threadIdx.x; e < kC * 64 / w; e += 256) {
            const int j = e / (64 / w), x = (e % (64 / w)) * w;
            const bool ok = j < nt && c0 + x < dv;
            cp_async(&Vs[j][x], vrow + (ok ? (int64_t)j * C + c0 + x : 0), ok, wide_v);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    issue_values(0);
    __syncthreads();
    // ---- B in two halves of 32: the diagonal blocks column by column (a lane per column, everything in registers), then B21 = -B22 M21 B11 --------------
    if (warp < 2) {
        const int o = warp * 32;
        float a[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) a[i] = i == lane ? 1.f : 0.f;
#pragma unroll
        for (int s = 0; s < 32; ++s) {
            const float u = bs[o + s] * a[s];
            Bt[o + lane][o + s] = u;                           // B[s][column] stored at [column][row]
#pragma unroll
            for (int i4 = (s + 1) >> 2; i4 < 8; ++i4) {
                const float4 m = *reinterpret_cast<const float4*>(&Mt[o + s][o + 4 * i4]);
                if (4 * i4 > s) a[4 * i4] = fmaf(-m.x, u, a[4 * i4]);
                if (4 * i4 + 1 > s) a[4 * i4 + 1] = fmaf(-m.y, u, a[4 * i4 + 1]);
                if (4 * i4 + 2 > s) a[4 * i4 + 2] = fmaf(-m.z, u, a[4 * i4 + 2]);
                a[4 * i4 + 3] = fmaf(-m.w, u, a[4 * i4 + 3]);
            }
        }
    }
    __syncthreads();
    {
        // X = M21 B11, X[t][j] kept at Mt[32 + j][t]: the quarter of the tile that would hold scores over later tokens
        const int t = threadIdx.x & 31, j0 = (threadIdx.x >> 5) * 4;
        float x[4] = {0.f, 0.f, 0.f, 0.f};
        for (int s = 0; s < 32; ++s) {
            const float m = Mt[s][32 + t];
#pragma unroll
            for (int l = 0; l < 4; ++l) x[l] = fmaf(m, Bt[j0 + l][s], x[l]);
        }
        __syncthreads();
#pragma unroll
        for (int l = 0; l < 4; ++l) Mt[32 + j0 + l][t] = x[l];
        __syncthreads();
        float y[4] = {0.f, 0.f, 0.f, 0.f};
        for (int s = 0; s < 32; ++s) {
            const float m = Bt[32 + s][32 + t];                // B22[t][s]
#pragma unroll
            for (int l = 0; l < 4; ++l) y[l] = fmaf(-m, Mt[32 + j0 + l][s], y[l]);
        }
#pragma unroll
        for (int l = 0; l < 4; ++l) { Bt[j0 + l][32 + t] = y[l]; Bt[32 + j0 + l][t] = 0.f; }
    }
    // ---- W = B K_P and U0 = B V: rows ty * 4 .., columns tx * 4 .. of 64 at a time --------------------------------------------------------------------------
    auto product = [&](const float* right, int pitch, float (&acc)[4][4]) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int l = 0; l < 4; ++l) acc[i][l] = 0.f;
        const int last = ty * 4 + 4;
#pragma unroll 4
        for (int s = 0; s < last; ++s) {
            const float4 bv = *reinterpret_cast<const float4*>(&Bt[s][ty * 4]), rv = *reinterpret_cast<const float4*>(right + s * pitch + tx * 4);
            const float bb[4] = {bv.x, bv.y, bv.z, bv.w}, rr[4] = {rv.x, rv.y, rv.z, rv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int l = 0; l < 4; ++l) acc[i][l] = fmaf(bb[i], rr[l], acc[i][l]);
        }
    };
    auto store = [&](float* base, int n, int c0, const float (&acc)[4][4]) {     // rows of n entries per (token, head)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int t = ty * 4 + i, cc = c0 + tx * 4;
            if (t >= nt || cc >= n) continue;
            float* dst = base + ((int64_t)(tf + t) * H + h) * n + cc;
            if ((n & 3) == 0) { *reinterpret_cast<float4*>(dst) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]); continue; }
#pragma unroll
            for (int l = 0; l < 4; ++l)
                if (cc + l < n) dst[l] = acc[i][l];
        }
    };
    __syncthreads();
    float acc[4][4];
    for (int c0 = 0; c0 < dk; c0 += 64) {
        if (kKD >= 64 || tx < 8) { product(KP + c0, kKp, acc); store(A.W, dk, c0, acc); }
    }
    for (int c0 = 0; c0 < dv; c0 += 64) {
        if (c0 > 0) { __syncthreads(); issue_values(c0); }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        product(&Vs[0][0], kLd, acc);
        store(A.U, dv, c0, acc);
    }
}

// ---- the walk ------------------------------------------------------------------------------------------------------------------------------------------
constexpr int kVB = 16, kVp = 20;                // value columns of a block and their pitch

constexpr int kWalkThreads = 512;
template <int kKD> constexpr int walk_stage_floats() { return 2 * kC * (kKD + 4) + kC * kVp + kKD; }
template <int kKD> constexpr int walk_red_floats() {          // partial sums: of the first product per share of the key rows, of the update per share of the tokens
    constexpr int a = (kWalkThreads / 64) * kC * kVp, b = (kWalkThreads / kKD) * kKD * kVp;
    return a > b ? a : b;
}
template <int kKD> constexpr int walk_floats() { return 2 * walk_stage_floats<kKD>() + walk_red_floats<kKD>() + kC * kVp + kKD * kVp; }

template <int kKD>
__global__ void __launch_bounds__(kWalkThreads)
delta_chunk_walk_kernel(const DeltaChunkArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr int kKp = kKD + 4, kStage = walk_stage_floats<kKD>();
    constexpr int kKG = kWalkThreads / 64, kKs = kKD / kKG;            // first product: shares of the key rows and their size
    constexpr int kRG = kKD / 4, kSG = kWalkThreads / (4 * kRG), kTs = kC / kSG;      // update: groups of four key rows, shares of the tokens and their size
    static_assert(kKs % 4 == 0 && kTs * kSG == kC, "shares of whole fours");
    extern __shared__ __align__(16) float sm[];
    float* red = sm + 2 * kStage;                                      // [kKG][64][20] / [kSG][kKD][20]
    float* Us = red + walk_red_floats<kKD>();                          // [64][20]
    float* S = Us + kC * kVp;                                          // [kKD][20]
    const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * kVB;
    const int t0 = A.cu[b], rows = A.cu[b + 1] - t0;
    if (rows <= 0) return;
    const int dk = A.dk, dv = A.dv, H = A.H, nc = (rows + kC - 1) / kC, base = chunk_base(A.cu, b);
    const int tid = threadIdx.x;
    const bool wide_k = (dk & 3) == 0, wide_v = (dv & 3) == 0;
    auto issue = [&](int c, int stage) {                               // one chunk's W, R k rows, U0 columns and decay product on their way to shared memory
        float* Ws = sm + stage * kStage;
        float* Ks = Ws + kC * kKp;
        float* U0 = Ks + kC * kKp;
        float* Pe = U0 + kC * kVp;
        const int tf = t0 + c * kC, nt = min(kC, rows - c * kC);
        const float* Wg = A.W + ((int64_t)tf * H + h) * dk;
        const float* Kg = A.KE + ((int64_t)tf * H + h) * dk;
        const int ek = wide_k ? 4 : 1, ev = wide_v ? 4 : 1, ld = H * dk;
        for (int e = tid; e < kC * kKD / ek; e += kWalkThreads) {
            const int j = e / (kKD / ek), r = (e % (kKD / ek)) * ek;
            const bool ok = j < nt && r < dk;
            const int at = ok ? j * ld + r : 0;
            cp_async(Ws + j * kKp + r, Wg + at, ok, wide_k);
            cp_async(Ks + j * kKp + r, Kg + at, ok, wide_k);
        }
        const float* Ug = A.U + ((int64_t)tf * H + h) * dv;
        for (int e = tid; e < kC * kVB / ev; e += kWalkThreads) {
            const int j = e / (kVB / ev), x = (e % (kVB / ev)) * ev;
            const bool ok = j < nt && c0 + x < dv;
            cp_async(U0 + j * kVp + x, Ug + (ok ? j * H * dv + c0 + x : 0), ok, wide_v);
        }
        for (int e = tid; e < kKD / ek; e += kWalkThreads) {
            const int r = e * ek;
            const bool ok = r < dk;
            cp_async(Pe + r, A.Pe + ((int64_t)(base + c) * H + h) * dk + (ok ? r : 0), ok, wide_k);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    issue(0, 0);
    const bool fresh = A.start[b] == 0;
    float* Sg = A.state + ((int64_t)A.slots[b] * H + h) * dv * dk;
    for (int e = tid; e < kKD * kVB; e += kWalkThreads) {
        const int x = e / kKD, r = e % kKD;
        S[r * kVp + x] = (!fresh && r < dk && c0 + x < dv) ? Sg[(int64_t)(c0 + x) * dk + r] : 0.f;
    }
    // roles: first product -- column group cg, rows ig + 16 a, share kg of the key rows; update -- column group cg, key rows rg * 4 .., share sg of the tokens
    const int cg = tid & 3, ig = (tid >> 2) & 15, kg = tid >> 6, rg = (tid >> 2) % kRG, sg = (tid >> 2) / kRG;
    for (int c = 0; c < nc; ++c) {
        const int stage = c & 1, tf = t0 + c * kC, nt = min(kC, rows - c * kC);
        const float* Ws = sm + stage * kStage;
        const float* Ks = Ws + kC * kKp;
        const float* U0 = Ks + kC * kKp;
        const float* Pe = U0 + kC * kVp;
        if (c + 1 < nc) {
            issue(c + 1, stage ^ 1);                                   // that stage was last read before the barriers of the previous chunk's update
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        // the state entering this chunk, for the outputs
        float* Sc = A.Sc + ((int64_t)(base + c) * H + h) * dv * dk + c0;
        for (int e = tid; e < kKD * 4; e += kWalkThreads) {
            const int r = e >> 2, x = (e & 3) * 4;
            if (r >= dk) continue;
            const float4 v = *reinterpret_cast<const float4*>(S + r * kVp + x);
            float* dst = Sc + (int64_t)r * dv + x;
            if (wide_v) { if (c0 + x < dv) *reinterpret_cast<float4*>(dst) = v; continue; }
            const float vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int l = 0; l < 4; ++l)
                if (c0 + x + l < dv) dst[l] = vv[l];
        }
        float acc[4][4] = {};
#pragma unroll
        for (int k = kg * kKs; k < (kg + 1) * kKs; k += 4) {
            float4 s4[4], w4[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                s4[i] = *reinterpret_cast<const float4*>(S + (k + i) * kVp + cg * 4);
                w4[i] = *reinterpret_cast<const float4*>(Ws + (ig + 16 * i) * kKp + k);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float w[4] = {w4[i].x, w4[i].y, w4[i].z, w4[i].w};
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc[i][0] = fmaf(w[j], s4[j].x, acc[i][0]); acc[i][1] = fmaf(w[j], s4[j].y, acc[i][1]);
                    acc[i][2] = fmaf(w[j], s4[j].z, acc[i][2]); acc[i][3] = fmaf(w[j], s4[j].w, acc[i][3]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(red + (kg * kC + ig + 16 * i) * kVp + cg * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        __syncthreads();
        if (tid < kC * 4) {
            const int j = tid >> 2, x = (tid & 3) * 4;
            float4 u = *reinterpret_cast<const float4*>(U0 + j * kVp + x);
#pragma unroll
            for (int q = 0; q < kKG; ++q) {
                const float4 r = *reinterpret_cast<const float4*>(red + (q * kC + j) * kVp + x);
                u.x -= r.x; u.y -= r.y; u.z -= r.z; u.w -= r.w;
            }
            *reinterpret_cast<float4*>(Us + j * kVp + x) = u;
            if (j < nt) {
                float* dst = A.U + ((int64_t)(tf + j) * H + h) * dv + c0 + x;
                if (wide_v) { if (c0 + x < dv) *reinterpret_cast<float4*>(dst) = u; }
                else {
                    const float uu[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
                    for (int l = 0; l < 4; ++l)
                        if (c0 + x + l < dv) dst[l] = uu[l];
                }
            }
        }
        __syncthreads();
        float up[4][4] = {};
#pragma unroll 8
        for (int s = sg * kTs; s < (sg + 1) * kTs; ++s) {
            const float4 k4 = *reinterpret_cast<const float4*>(Ks + s * kKp + rg * 4), u4 = *reinterpret_cast<const float4*>(Us + s * kVp + cg * 4);
            const float k[4] = {k4.x, k4.y, k4.z, k4.w}, u[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int l = 0; l < 4; ++l) up[i][l] = fmaf(k[i], u[l], up[i][l]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(red + (sg * kKD + rg * 4 + i) * kVp + cg * 4) = make_float4(up[i][0], up[i][1], up[i][2], up[i][3]);
        __syncthreads();
        for (int e = tid; e < kKD * 4; e += kWalkThreads) {
            const int r = e >> 2, x = (e & 3) * 4;
            float4 s = *reinterpret_cast<const float4*>(S + r * kVp + x);
            const float pe = Pe[r];
            s.x *= pe; s.y *= pe; s.z *= pe; s.w *= pe;
#pragma unroll
            for (int q = 0; q < kSG; ++q) {
                const float4 v = *reinterpret_cast<const float4*>(red + (q * kKD + r) * kVp + x);
                s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
            }
            *reinterpret_cast<float4*>(S + r * kVp + x) = s;
        }
        __syncthreads();
    }
    for (int e = tid; e < kKD * kVB; e += kWalkThreads) {
        const int x = e / kKD, r = e % kKD;
        if (r < dk && c0 + x < dv) Sg[(int64_t)(c0 + x) * dk + r] = S[r * kVp + x];
    }
}

// ---- the outputs ---------------------------------------------------------------------------------------------------------------------------------------
template <int kW> constexpr int out_floats() { return 2 * 32 * (kLd + kW + 4) + kC * kLd + kC * (kW + 4); }

// kW: value columns of a block (64 or 128); a thread makes four tokens x kW / 16 columns (groups of four, 64 columns apart).  All operands arrive by cp.async as they lie:
// slabs of 32 key rows of P q and of the entering state (two buffers), N and u for the second term under the first one.
template <int kW>
__global__ void __launch_bounds__(256, 2)
delta_chunk_output_kernel(const DeltaChunkArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr int kWp = kW + 4, kGr = kW / 64, kSlab = 32 * (kLd + kWp);
    extern __shared__ __align__(16) float sm[];             // two slabs: [32][68] P q, [32][kWp] state
    float* ns = sm + 2 * kSlab;                             // [64][68] N: [s][t]
    float* us = ns + kC * kLd;                              // [64][kWp] u: [s][column]
    const int h = blockIdx.y, b = blockIdx.z / A.max_chunks, c = blockIdx.z % A.max_chunks;
    const int t0 = A.cu[b], rows = A.cu[b + 1] - t0;
    if (c * kC >= rows) return;
    const int tf = t0 + c * kC, nt = min(kC, rows - c * kC);
    const int dk = A.dk, dv = A.dv, H = A.H, c0 = blockIdx.x * kW;
    const int64_t ch = (int64_t)(chunk_base(A.cu, b) + c) * H + h;
    const float* Sc = A.Sc + ch * dv * dk + c0;
    const float* QPt = A.QP + ch * dk * kC;
    const float* Nt = A.N + ch * kC * kC;
    const float* Ug = A.U + ((int64_t)tf * H + h) * dv + c0;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const bool wide_v = (dv & 3) == 0;
    const int ev = wide_v ? 4 : 1;
    auto issue = [&](int r0, int stage) {
        float* qs = sm + stage * kSlab;
        float* ss = qs + 32 * kLd;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int x = (threadIdx.x >> 4) + 16 * i, t = tx * 4;
            const bool ok = r0 + x < dk;
            cp_async(qs + x * kLd + t, QPt + (ok ? (r0 + x) * kC + t : 0), ok, true);
        }
        for (int e = threadIdx.x; e < 32 * kW / ev; e += 256) {
            const int x = e / (kW / ev), k = (e % (kW / ev)) * ev;
            const bool ok = r0 + x < dk && c0 + k < dv;
            cp_async(ss + x * kWp + k, Sc + (ok ? (int64_t)(r0 + x) * dv + k : 0), ok, wide_v);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    issue(0, 0);
    for (int e = threadIdx.x; e < kC * 16; e += 256) cp_async(ns + (e >> 4) * kLd + (e & 15) * 4, Nt + e * 4, true, true);
    for (int e = threadIdx.x; e < kC * kW / ev; e += 256) {
        const int j = e / (kW / ev), k = (e % (kW / ev)) * ev;
        const bool ok = j < nt && c0 + k < dv;
        cp_async(us + j * kWp + k, Ug + (ok ? (int64_t)j * H * dv + k : 0), ok, wide_v);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    float o[4][4 * kGr] = {};
    auto multiply = [&](const float* left, const float* right) {       // one term: four tokens' factors times the columns' row
        const float4 l4 = *reinterpret_cast<const float4*>(left);
        const float l[4] = {l4.x, l4.y, l4.z, l4.w};
#pragma unroll
        for (int g = 0; g < kGr; ++g) {
            const float4 r4 = *reinterpret_cast<const float4*>(right + 64 * g);
            const float r[4] = {r4.x, r4.y, r4.z, r4.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int k = 0; k < 4; ++k) o[i][4 * g + k] = fmaf(l[i], r[k], o[i][4 * g + k]);
        }
    };
    for (int r0 = 0, stage = 0; r0 < dk; r0 += 32, stage ^= 1) {
        const bool first = r0 == 0, more = r0 + 32 < dk;
        if (more) issue(r0 + 32, stage ^ 1);
        // the slab in use is the oldest group but one (N and u were asked for right after the first slab)
        if (first) { if (more) asm volatile("cp.async.wait_group 2;" ::: "memory"); else asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else { if (more) asm volatile("cp.async.wait_group 1;" ::: "memory"); else asm volatile("cp.async.wait_group 0;" ::: "memory"); }
        __syncthreads();
        const float* qs = sm + stage * kSlab + ty * 4;
        const float* ss = sm + stage * kSlab + 32 * kLd + tx * 4;
#pragma unroll 8
        for (int k = 0; k < 32; ++k) multiply(qs + k * kLd, ss + k * kWp);
        __syncthreads();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int last = min(nt, ty * 4 + 4);
#pragma unroll 4
    for (int k = 0; k < last; ++k) multiply(ns + k * kLd + ty * 4, us + k * kWp + tx * 4);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty * 4 + i;
        if (t >= nt) continue;
#pragma unroll
        for (int g = 0; g < kGr; ++g) {
            const int cv = c0 + 64 * g + tx * 4;
            float* dst = A.out + ((int64_t)(tf + t) * H + h) * dv + cv;
            if ((dv & 3) == 0) { if (cv < dv) *reinterpret_cast<float4*>(dst) = make_float4(o[i][4 * g], o[i][4 * g + 1], o[i][4 * g + 2], o[i][4 * g + 3]); continue; }
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (cv + k < dv) dst[k] = o[i][4 * g + k];
        }
    }
}

int64_t round4(int64_t n) { return (n + 3) & ~(int64_t)3; }

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int64_t gated_delta_channel_chunked_scratch(int32_t num_tokens, int32_t num_seqs, int32_t num_heads, int32_t dk, int32_t dv) {
    const int64_t th = (int64_t)num_tokens * num_heads, sh = chunk_slots(num_tokens, num_seqs) * num_heads;
    return 2 * round4(th * dk) + sh * dk * kC + sh * kC * kC + round4(th * dv) + round4(sh * dk) + round4(sh * dv * dk);
}

void gated_delta_channel_chunked(const float* qkv, const float* proj, int64_t ld_proj, int32_t off_b, const float* decay, float* state, float* out, float* scratch,
                                 const int32_t* cu_seqlens, const int32_t* seq_slots, const int32_t* seq_start, int32_t num_tokens, int32_t num_seqs, int32_t max_rows,
                                 int32_t num_heads, int32_t num_kv_heads, int32_t dk, int32_t dv, int64_t stream) {
    if (num_seqs == 0 || num_tokens == 0) return;
    B200_REQUIRE(qkv && proj && decay && state && out && scratch && cu_seqlens && seq_slots && seq_start, kErrBadArg, "gated_delta_channel_chunked: null pointer");
    B200_REQUIRE(num_heads > 0 && num_heads <= 65535 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dk > 0 && dv > 0 && max_rows > 0 && num_seqs <= 65535, kErrBadArg,
                 "gated_delta_channel_chunked: bad sizes");
    B200_REQUIRE((((uintptr_t)scratch | (uintptr_t)out) & 15) == 0, kErrBadArg, "gated_delta_channel_chunked: scratch and out start on 16-byte borders");
    B200_REQUIRE(dk <= 128, kErrUnsupported, "gated_delta_channel_chunked: key size %d > 128", dk);
    const int max_chunks = (max_rows + kC - 1) / kC;
    B200_REQUIRE((int64_t)max_chunks * num_seqs <= 65535, kErrUnsupported, "gated_delta_channel_chunked: %d chunks x %d entries exceed the grid", max_chunks, num_seqs);
    const int64_t th = (int64_t)num_tokens * num_heads, sh = chunk_slots(num_tokens, num_seqs) * num_heads;
    DeltaChunkArgs A{qkv, proj, ld_proj, off_b, decay, state, out, cu_seqlens, seq_slots, seq_start, num_tokens, num_heads, num_kv_heads, dk, dv, max_chunks,
                     nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr};
    A.W = scratch;
    A.KE = A.W + round4(th * dk);
    A.QP = A.KE + round4(th * dk);
    A.N = A.QP + sh * dk * kC;
    A.U = A.N + sh * kC * kC;
    A.Pe = A.U + round4(th * dv);
    A.Sc = A.Pe + round4(sh * dk);
    cudaStream_t st = as_stream(stream);
    const unsigned z = (unsigned)(max_chunks * num_seqs);
#define DCH(KD) do { \
        const int s1 = kPrepFloats(KD) * (int)sizeof(float), s2 = walk_floats<KD>() * (int)sizeof(float); \
        ensure_dynamic_smem(reinterpret_cast<const void*>(delta_chunk_prepare_kernel<KD>), s1); \
        ensure_dynamic_smem(reinterpret_cast<const void*>(delta_chunk_walk_kernel<KD>), s2); \
        launch_pdl(delta_chunk_prepare_kernel<KD>, dim3(1, num_heads, z), dim3(256), (size_t)s1, st, A); \
        launch_pdl(delta_chunk_walk_kernel<KD>, dim3(ceil_div(dv, kVB), num_heads, num_seqs), dim3(kWalkThreads), (size_t)s2, st, A); } while (0)
    if (dk <= 32) DCH(32);
    else if (dk <= 64) DCH(64);
    else DCH(128);
#undef DCH
#define DCO(W) do { \
        const int s3 = out_floats<W>() * (int)sizeof(float); \
        ensure_dynamic_smem(reinterpret_cast<const void*>(delta_chunk_output_kernel<W>), s3); \
        launch_pdl(delta_chunk_output_kernel<W>, dim3(ceil_div(dv, W), num_heads, z), dim3(256), (size_t)s3, st, A); } while (0)
    if (dv <= 64) DCO(64);
    else DCO(128);
#undef DCO
    count_launch(3);
    check_launch("gated_delta_channel_chunked");
}

}  // extern "C"
